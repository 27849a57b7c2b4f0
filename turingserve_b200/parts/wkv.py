"""Time mixer with a matrix state per head that fades channel by channel at rates the token chooses (the sixth generation of
RWKV; Peng et al., "Eagle and Finch: RWKV with Matrix-Valued States and Dynamic Recurrence").

With h' the token's predecessor (zeros before the first), r, k, v, the gate and the decay each read a mix of their own,
h + (h' - h) mu ('mu.r', ...).  r, k, v and the gate are products of their mixes ('r', 'k', 'v', 'g'); the decay is
w = exp(-exp(W_w2 tanh(W_w1 mix) + w0)) per head and key channel ('w1', 'w2', 'w0'), in 32-bit after the first product.  Per
head, in 32-bit, with the bonus u for the present token only:
    o = (S + diag(u) k v^T)^T r,    S <- diag(w) S + k v^T.
Every head's o is divided by its root mean square, scaled by a weight ('norm'), gated by silu; then the output projection.

Nothing is cached per token.  The mixer declares one flat 32-bit state per request, [H D D values of S | the last input],
zeroed when the request is admitted, so the first portion needs no branch and a captured step's padding rows update the null
slot.  The rank of the decay's two products is whatever the checkpoint has.
"""

from __future__ import annotations

import torch

from turingserve_b200 import kernels
from turingserve_b200.parts.base import BuildContext, Mixer, ParamSpec, StateNeed, register

MIXES = ("r", "k", "v", "g", "w")
PROJECTIONS = ("r", "k", "v", "g")


class WKV(Mixer):
    MAX_DIM = 256               # the scan's limit on a head's width
    RANDOM_RANK = 64            # the decay's rank in the random-weights mode where the spec names none

    def __init__(self, spec, ctx: BuildContext) -> None:
        self.hidden = ctx.hidden_size
        self.H, self.D = int(spec.num_heads), int(spec.head_dim)
        if self.H < 1 or not 1 <= self.D <= self.MAX_DIM:
            raise ValueError(f"wkv: {self.H} heads of {self.D} (the kernels take heads of up to {self.MAX_DIM})")
        self.eps = float(spec.norm_eps)
        self.rank = None if spec.decay_rank is None else int(spec.decay_rank)
        # (the last input starts on a 16-byte boundary of the slot)
        self.prev_off = self.H * self.D * self.D
        self.mu = self.w = self.w1 = self.w2 = self.w0 = self.u = self.norm_w = self.w_o = None

    def parameters(self) -> dict[str, ParamSpec]:
        h, n = self.hidden, self.H * self.D
        free = self.rank or self.RANDOM_RANK
        p = {f"mu.{s}": ParamSpec((h,)) for s in MIXES}
        p.update({s: ParamSpec((n, h)) for s in PROJECTIONS})
        p.update({"w1": ParamSpec((self.rank, h), free=free), "w2": ParamSpec((n, self.rank), free=free),
                  "w0": ParamSpec((n,), compute_dtype=False), "u": ParamSpec((self.H, self.D), compute_dtype=False),
                  "norm": ParamSpec((n,), compute_dtype=False, init="ones"), "o": ParamSpec((h, n))})
        return p

    def load(self, t: dict[str, torch.Tensor]) -> None:
        if t["w1"].shape[0] != t["w2"].shape[1]:
            raise ValueError(f"wkv: w1 has {t['w1'].shape[0]} rows, w2 {t['w2'].shape[1]} columns")
        self.mu = torch.stack([t[f"mu.{s}"] for s in MIXES]).contiguous()
        self.w = torch.stack([t[s] for s in PROJECTIONS]).contiguous()
        self.w1, self.w2, self.w_o = t["w1"].contiguous(), t["w2"].contiguous(), t["o"].contiguous()
        self.w0, self.u = t["w0"].float().contiguous(), t["u"].float().contiguous()
        self.norm_w = t["norm"].float().contiguous()

    def state_need(self) -> StateNeed:
        # (padded to whole 16 bytes, so that every slot's last input starts on such a boundary where H D D does)
        return StateNeed((-(-(self.prev_off + self.hidden) // 4) * 4,), torch.float32)

    def forward(self, x: torch.Tensor, step, cache, state: torch.Tensor) -> torch.Tensor:
        ops = kernels.ops()
        T, H, D, n = x.shape[0], self.H, self.D, self.H * self.D
        new = lambda *shape, dtype=x.dtype: torch.empty(shape, dtype=dtype, device=x.device)
        rkvg = new(4, T, n)
        z = new(T, self.w1.shape[0], dtype=torch.float32)
        if not ops.wkv_project(rkvg, z, x, self.mu, self.w, self.w1, state, self.prev_off, step):
            mixes = new(5, T, self.hidden)
            ops.token_shift(mixes, x, self.mu, state, self.prev_off, step)
            for i in range(4):
                ops.linear(rkvg[i], mixes[i], self.w[i])
            ops.linear(z, mixes[4], self.w1)
        y = new(T, n)
        if not ops.wkv_step(y, rkvg, z, self.w2, self.w0, self.u, self.norm_w, self.eps, x, state, step, H, D):
            w = new(T, n, dtype=torch.float32)
            ops.wkv_decay(w, z, self.w2, self.w0)
            o = new(T, n, dtype=torch.float32)
            ops.wkv_scan(o, rkvg[0], rkvg[1], rkvg[2], w, self.u, x, state, step, H, D)
            ops.head_gated_rmsnorm(y, o, rkvg[3], self.norm_w, self.eps, H, D)
        return ops.linear(new(T, self.hidden), y, self.w_o, may_defer=True)


register("mixer", "wkv", WKV)
