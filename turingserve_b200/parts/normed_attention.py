"""Grouped-query attention with norms on q, k and v, capped scores, a window that keeps the first tokens, values that
carry their positions, and a gate per head, over the paged cache.

One fused projection gives, per token, [q (H D) | k (G D) | v (G V) | gate (H)]; no biases.  Every head of q and k is
RMS-normed over its D dimensions (learned weights 'q.norm' and 'k.norm', common to the heads), then rotated over its first
dimensions (the position encoding named in the spec: pairs (i, i + dims/2), angle = position * frequency in 32-bit, cosine
and sine times the encoding's magnitude).  Every head's value is divided by its root mean square (no weight) and turned
by its position over all its V dimensions, pairs (m, m + V/2); the cache keeps it so.  score = cap tanh(q.k scale / cap);
position i sees i - window < j <= i and the first ``keep_first`` positions; ordinary softmax.  A head's output at position i,
a sum of values turned by their own positions, is turned back by i, so that what it holds depends on distances only, and
multiplied by sigmoid of the head's gate, both on its way out of the attention kernel; output projection.  Norms, rotation,
turned values, cap, window and gate are each optional in the spec.
"""

from __future__ import annotations

import torch

from turingserve_b200 import kernels
from turingserve_b200.parts.base import BuildContext, CacheNeed, Mixer, ParamSpec, build, register


class NormedAttention(Mixer):
    MAX_KEY, MAX_VALUE = 1024, 512          # the any-size attention kernel's limits
    ROW_ALIGN = 8                           # the projection's rows start on 16-byte boundaries

    def __init__(self, spec, ctx: BuildContext) -> None:
        self.hidden = ctx.hidden_size
        self.H, self.G = int(spec.num_heads), int(spec.num_kv_heads)
        self.D, self.V = int(spec.key_dim), int(spec.value_dim)
        if self.G < 1 or self.H % self.G:
            raise ValueError("num_heads must be a multiple of num_kv_heads")
        if not (0 < self.D <= self.MAX_KEY and 0 < self.V <= self.MAX_VALUE):
            raise ValueError(f"normed_attention: keys of {self.D}, values of {self.V}: the kernels take up to "
                             f"{self.MAX_KEY} and {self.MAX_VALUE}")
        self.scale, self.eps = float(spec.scale), float(spec.norm_eps)
        self.softcap = float(spec.softcap) if spec.softcap else 0.0
        self.window = int(spec.window) if spec.window else None
        self.keep = int(spec.keep_first) if self.window else 0
        self.has_qk_norm, self.v_norm, self.has_gate = bool(spec.qk_norm), bool(spec.value_norm), bool(spec.head_gate)
        self.position = build("position", spec.position, ctx) if spec.position is not None else None
        self.rot_dims, self.magnitude = 0, 1.0
        if self.position is not None:
            if getattr(self.position, "pairing", None) != "halves" or not hasattr(self.position, "freq"):
                raise ValueError("normed_attention takes a position encoding of paired halves given by frequencies (kinds "
                                 "rope_half, yarn_pairs with pairing 'halves')")
            self.rot_dims = int(self.position.dims)
            self.magnitude = float(getattr(self.position, "magnitude", 1.0))
            if self.rot_dims > self.D:
                raise ValueError(f"normed_attention: {self.rot_dims} rotated dimensions of {self.D}")
        self.v_freq = None
        if spec.value_base is not None:
            if self.V % 2:
                raise ValueError(f"normed_attention: {self.V} value dimensions do not pair")
            m = torch.arange(self.V // 2, dtype=torch.float64)
            self.v_freq = (float(spec.value_base) ** (-2.0 * m / self.V)).to(torch.float32).to(ctx.device).contiguous()
        self.q_dim, self.k_dim, self.v_dim = self.H * self.D, self.G * self.D, self.G * self.V
        self.g_off = self.q_dim + self.k_dim + self.v_dim
        self.n_in = -(-(self.g_off + (self.H if self.has_gate else 0)) // self.ROW_ALIGN) * self.ROW_ALIGN
        self.w_in = self.w_o = self.q_w = self.k_w = None

    def parameters(self) -> dict[str, ParamSpec]:
        p = {"q": ParamSpec((self.q_dim, self.hidden)), "k": ParamSpec((self.k_dim, self.hidden)),
             "v": ParamSpec((self.v_dim, self.hidden)), "o": ParamSpec((self.hidden, self.H * self.V))}
        if self.has_qk_norm:
            p.update({"q.norm": ParamSpec((self.D,), compute_dtype=False, init="ones"),
                      "k.norm": ParamSpec((self.D,), compute_dtype=False, init="ones")})
        if self.has_gate:
            p["g"] = ParamSpec((self.H, self.hidden))
        return p

    def load(self, t: dict[str, torch.Tensor]) -> None:
        rows = [t["q"], t["k"], t["v"]] + ([t["g"]] if self.has_gate else [])
        pad = self.n_in - sum(r.shape[0] for r in rows)
        if pad:
            rows.append(torch.zeros((pad, self.hidden), dtype=t["q"].dtype, device=t["q"].device))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_o = t["o"].contiguous()
        if self.has_qk_norm:
            self.q_w, self.k_w = t["q.norm"].float().contiguous(), t["k.norm"].float().contiguous()

    def cache_need(self) -> CacheNeed:
        return CacheNeed(self.G, self.D, self.window, value_dim=self.V, keep_first=self.keep)

    def forward(self, x: torch.Tensor, step, cache, state=None) -> torch.Tensor:
        ops = kernels.ops()
        T = x.shape[0]
        H, G, D, V = self.H, self.G, self.D, self.V
        grp = step.groups[cache.group]
        proj = torch.empty((T, self.n_in), dtype=x.dtype, device=x.device)
        # (a few tokens: the product's partial sums are summed by the kernel that norms and rotates them)
        proj = ops.linear(proj, x, self.w_in, may_defer=True, lazy=False)
        proj = ops.qkv_heads_write(proj, self.q_dim, self.q_dim + self.k_dim, step.positions, self.q_w, self.k_w, self.eps,
                                   self.position.freq if self.rot_dims else None, self.magnitude, self.rot_dims, self.v_norm,
                                   self.v_freq, cache.k, cache.v, grp.slot_mapping if cache.writable else None, H, G, D, V,
                                   cache.page_size)
        heads = torch.empty((T, H, V), dtype=x.dtype, device=x.device)
        gate = proj[:, self.g_off:self.g_off + H] if self.has_gate else None
        ops.attention_biased(heads, proj[:, :self.q_dim].view(T, H, D), cache.k, cache.v, grp.block_tables, step, G,
                             cache.page_size, self.scale, self.softcap, None, self.window, keep=self.keep,
                             out_freq=self.v_freq, gate=gate)
        out = torch.empty((T, self.hidden), dtype=x.dtype, device=x.device)
        return ops.linear(out, heads.view(T, H * V), self.w_o, may_defer=True)


register("mixer", "normed_attention", NormedAttention)
