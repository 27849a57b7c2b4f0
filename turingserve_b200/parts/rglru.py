"""Recurrent block of a real-gated linear recurrent unit (Griffin; De et al., "Griffin: Mixing Gated Linear Recurrences
with Local Attention for Efficient Language Models").

One fused projection gives, per token, [y (W) | x (W)] with biases.  u = causal filter of x, a few taps per channel
('conv' [W, taps], the last column the present token's, with bias 'conv.b', no activation).  u falls into ``num_blocks`` equal
parts; in part n r = sigmoid(ra[n] u + ra.b[n]) and i = sigmoid(ri[n] u + ri.b[n]), square matrices [out, in].  Per channel,
in 32-bit: log a = -scale r softplus(lam), S <- a S + sqrt(1 - a^2) i u.  Output: W_o (S gelu_tanh(y)).

Nothing is cached per token.  The mixer declares one flat 32-bit state per request, [W values of S | ring of taps x W
filter inputs, the one of position p in place p % taps], zeroed when the request is admitted, so the first portion needs no
branch and a captured step's padding rows update the null slot.
"""

from __future__ import annotations

import torch

from turingserve_b200 import kernels
from turingserve_b200.parts.base import BuildContext, Mixer, ParamSpec, StateNeed, register


class RGLRU(Mixer):
    MAX_TAPS = 8

    def __init__(self, spec, ctx: BuildContext) -> None:
        self.hidden = ctx.hidden_size
        self.W, self.blocks, self.taps = int(spec.width), int(spec.num_blocks), int(spec.conv_taps)
        self.decay_scale = float(spec.decay_scale)
        if self.blocks < 1 or self.W < 1 or self.W % self.blocks:
            raise ValueError(f"rglru: {self.W} channels do not fall into {self.blocks} equal parts")
        if not 1 <= self.taps <= self.MAX_TAPS:
            raise ValueError(f"rglru: a filter of {self.taps} taps (the kernels take 1 to {self.MAX_TAPS})")
        self.w_in = self.b_in = self.w_o = self.conv = self.conv_b = None
        self.ra = self.ri = self.ra_b = self.ri_b = self.rate = None

    def parameters(self) -> dict[str, ParamSpec]:
        W, n = self.W, self.blocks
        size = W // n
        p = {}
        for branch in ("y", "x"):
            p[branch] = ParamSpec((W, self.hidden))
            p[branch + ".b"] = ParamSpec((W,), init="zeros")
        p.update({"conv": ParamSpec((W, self.taps), compute_dtype=False),
                  "conv.b": ParamSpec((W,), compute_dtype=False, init="zeros")})
        for gate in ("ra", "ri"):
            p[gate] = ParamSpec((n, size, size))
            p[gate + ".b"] = ParamSpec((n, size), compute_dtype=False, init="zeros")
        p.update({"lam": ParamSpec((W,), compute_dtype=False), "o": ParamSpec((self.hidden, W))})
        return p

    def load(self, t: dict[str, torch.Tensor]) -> None:
        self.w_in = torch.cat([t["y"], t["x"]], dim=0).contiguous()
        self.b_in = torch.cat([t["y.b"], t["x.b"]]).contiguous()
        self.w_o = t["o"].contiguous()
        self.conv, self.conv_b = t["conv"].float().contiguous(), t["conv.b"].float().contiguous()
        self.ra, self.ri = t["ra"].contiguous(), t["ri"].contiguous()
        self.ra_b, self.ri_b = t["ra.b"].float().reshape(-1).contiguous(), t["ri.b"].float().reshape(-1).contiguous()
        # what multiplies r in -log a; worked out in double, rounded once
        self.rate = (self.decay_scale * torch.nn.functional.softplus(t["lam"].double(), threshold=40.0)).float().contiguous()

    def state_need(self) -> StateNeed:
        return StateNeed(((1 + (self.taps if self.taps > 1 else 0)) * self.W,), torch.float32)

    def forward(self, x: torch.Tensor, step, cache, state: torch.Tensor) -> torch.Tensor:
        ops = kernels.ops()
        T, W = x.shape[0], self.W
        proj = torch.empty((T, 2 * W), dtype=x.dtype, device=x.device)
        ops.linear(proj, x, self.w_in, self.b_in)
        s = torch.empty((T, W), dtype=x.dtype, device=x.device)
        if not ops.rglru_step(s, proj, 0, W, self.conv, self.conv_b, self.ra, self.ri, self.ra_b, self.ri_b, self.rate, state,
                              step, self.taps):
            u = torch.empty((T, W), dtype=x.dtype, device=x.device)
            ops.short_filter(u, proj, W, self.conv, self.conv_b, state, W, step, self.taps)
            ab = torch.empty((T, W, 2), dtype=torch.float32, device=x.device)
            ops.rglru_gates(ab, u, self.ra, self.ri, self.ra_b, self.ri_b, self.rate)
            ops.rglru_scan(s, ab, proj, 0, W, state, step, self.taps)
        out = torch.empty((T, self.hidden), dtype=x.dtype, device=x.device)
        return ops.linear(out, s, self.w_o, may_defer=True)


register("mixer", "rglru", RGLRU)
