"""Routed feed-forward: every token goes through the ``top_k`` of ``num_experts`` small feed-forwards
down_e(act(up_e(.))), or gated ones down_e(act(gate_e(.)) * up_e(.)), whose router scores are largest.
A learned correction may enter the choice (score + correction) without entering the weights.  The router may have
more outputs than there are experts with tensors: the outputs behind them are experts that return their input,
which cost no product (their pairs are sorted behind the others and the sum takes the token's own row for them).

A shared expert (``shared_intermediate_size``: one more feed-forward of the experts' form under 'shared.') runs for every
token and is added in the kernel that sums a token's choices, unweighted or (``shared_gate``) times sigmoid(W_sg x), one number
a token, which the router's kernel works out beside its scores.
With ``groups`` the experts fall into equal groups of neighbours, and only those of the ``groups_kept`` groups whose two largest
choice scores have the largest sums may be chosen.  ``weight_scale`` multiplies the weights.

Router logits and scores are 32-bit.  The (token, choice) pairs are sorted by expert on the device and the
two products run over the sorted groups; the chosen score multiplies the expert's input (``weight_on``
"input", the product reads score * x rounded to the engine's type) or its output; a token's choices are
summed in 32-bit in the order of their rank.  No count comes back to the host, so the chain may sit in a
captured step.  The experts' weights are stacked [E, ff, hidden] and [E, hidden, ff] when they arrive.

Many rows (``LIBRARY_ROWS`` pairs or more, outside a capture): the group sizes are read back once, the input
rows are gathered in sorted order, and every expert's rows go through ``ops().linear`` as a product of their own,
i.e. to the many-row kernels and the vendor library that the dense products of such steps use.  (With a table the host
counts the groups itself from the step's ids, and nothing is read back.)

Without a router (``table_rows``): an integer table ('table' [ids, top_k]) gives every token id its experts; the choices
weigh 1 / top_k each, and the sort reads the table itself, so neither router scores nor weights exist.

Gated experts: silu(gate) * up, or the clamped gated unit ("clamped_glu"), whose gate and up rows take turns in the stacked
weights: neighbouring columns of the first product are a gate and its up, and the grouped product's epilogue makes one
output of the two.
"""

from __future__ import annotations

import numpy as np
import torch

from turingserve_b200 import kernels
from turingserve_b200.parts.base import BuildContext, FeedForward, ParamSpec, RoutedSum, register
from turingserve_b200.parts.mlp import ACTIVATIONS


class RoutedMLP(FeedForward):
    # from this many (token, choice) pairs in a step the experts' products are launched one by one (2,048 tokens of
    # width 3,584 through 8 experts of 7,104: 2.7 ms for the two grouped products, 0.5 ms this way)
    LIBRARY_ROWS = 1024

    def __init__(self, spec, ctx: BuildContext) -> None:
        self.hidden = ctx.hidden_size
        self.E, self.top, self.inter = int(spec.num_experts), int(spec.top_k), int(spec.intermediate_size)
        if self.top < 1 or self.E < 0:
            raise ValueError(f"routed_mlp: top {self.top} of {self.E} experts")
        self.glu = spec.activation == "clamped_glu"
        if spec.activation not in ACTIVATIONS and not self.glu:
            raise ValueError(f"routed_mlp: activation {spec.activation!r} has no kernel")
        if spec.scoring not in ("sigmoid", "softmax") or spec.weight_on not in ("input", "output"):
            raise ValueError(f"routed_mlp: scoring {spec.scoring!r} / weight_on {spec.weight_on!r}")
        self.activation, self.softmax = spec.activation, spec.scoring == "softmax"
        self.renormalize, self.on_input = bool(spec.renormalize), spec.weight_on == "input"
        self.gated, self.has_correction = bool(getattr(spec, "gated", False)), bool(getattr(spec, "correction", False))
        self.identity = int(getattr(spec, "identity", 0))
        if self.identity < 0:
            raise ValueError(f"routed_mlp: {self.identity} identity experts")
        if self.glu and not self.gated:
            raise ValueError("routed_mlp: the clamped gated unit needs gated experts")
        if self.gated and self.activation != "silu" and not self.glu:
            raise ValueError(f"routed_mlp: gated experts with activation {self.activation!r} have no kernel")
        if self.identity and self.on_input:
            raise ValueError("routed_mlp: experts that return their input are weighted on the output")
        self.outputs = self.E + self.identity           # what the router scores
        if self.top > self.outputs:
            raise ValueError(f"routed_mlp: top {self.top} of {self.outputs} router outputs")
        shared = getattr(spec, "shared_intermediate_size", None)
        self.shared_inter = int(shared) if shared else 0
        self.groups, self.groups_kept = int(getattr(spec, "groups", 1)), int(getattr(spec, "groups_kept", 1))
        self.weight_scale, self.has_share = float(getattr(spec, "weight_scale", 1.0)), bool(getattr(spec, "shared_gate", False))
        if self.groups < 1 or self.outputs % self.groups or not 1 <= self.groups_kept <= self.groups:
            raise ValueError(f"routed_mlp: {self.groups_kept} of {self.groups} groups of {self.outputs} experts")
        if self.top > self.outputs // self.groups * self.groups_kept:
            raise ValueError(f"routed_mlp: top {self.top} of {self.groups_kept} groups of {self.outputs // self.groups} experts")
        if self.has_share and not self.shared_inter:
            raise ValueError("routed_mlp: a shared expert's gate without a shared expert")
        rows = getattr(spec, "table_rows", None)
        self.table_rows = int(rows) if rows else 0
        self.wants_step = self.table_rows > 0
        if self.table_rows and (self.has_correction or self.identity or self.on_input or self.E == 0 or self.groups > 1
                                or self.has_share or self.weight_scale != 1.0):
            raise ValueError("routed_mlp: a table of experts comes without router, correction, groups, shared gate and identity "
                             "outputs, its weights on the output")
        if self.glu:
            self.glu_args = (float(spec.glu_limit), float(spec.glu_slope), float(spec.glu_offset))
            self.shared_glu_args = (float(spec.shared_glu_limit), float(spec.glu_slope), float(spec.glu_offset))
        self.table = self.host_table = None
        self.w_router = self.w_up = self.w_down = self.correction = self.w_shared_up = self.w_shared_down = None

    def parameters(self) -> dict[str, ParamSpec]:
        if self.table_rows:
            p = {"table": ParamSpec((self.table_rows, self.top), integer=True, init="distinct", high=self.E)}
        else:
            p = {"router": ParamSpec((self.outputs, self.hidden), compute_dtype=False)}
        if self.has_correction:
            p["correction"] = ParamSpec((self.outputs,), compute_dtype=False, init="zeros")
        for e in range(self.E):
            if self.gated:
                p[f"e{e}.gate"] = ParamSpec((self.inter, self.hidden))
            p[f"e{e}.up"] = ParamSpec((self.inter, self.hidden))
            p[f"e{e}.down"] = ParamSpec((self.hidden, self.inter))
        if self.shared_inter:
            if self.gated:
                p["shared.gate"] = ParamSpec((self.shared_inter, self.hidden))
            p["shared.up"] = ParamSpec((self.shared_inter, self.hidden))
            p["shared.down"] = ParamSpec((self.hidden, self.shared_inter))
            if self.has_share:
                p["shared.sg"] = ParamSpec((1, self.hidden), compute_dtype=False)
        return p

    def load(self, t: dict[str, torch.Tensor]) -> None:
        if self.table_rows:
            self.table = t["table"].contiguous()
            self.host_table = self.table.cpu().numpy()
            lo, hi = int(self.table.min()), int(self.table.max())
            if lo < 0 or hi >= self.E:
                raise ValueError(f"routed_mlp: the table names experts {lo} to {hi} of {self.E}")
        else:
            # (the shared expert's gate is one more row of the router)
            rows = [t["router"].float()] + ([t["shared.sg"].float()] if self.has_share else [])
            self.w_router = torch.cat(rows, dim=0).contiguous()
        if self.has_correction:
            self.correction = t["correction"].float().contiguous()
        if self.shared_inter:
            self.w_shared_up = self._pack(t, "shared.")
            self.w_shared_down = t["shared.down"].contiguous()
        if self.E == 0:
            return
        # gated experts: an expert's gate rows, then its up rows, in one product
        self.w_up = torch.stack([self._pack(t, f"e{e}.") for e in range(self.E)]).contiguous()
        self.w_down = torch.stack([t[f"e{e}.down"] for e in range(self.E)]).contiguous()

    def _pack(self, t: dict[str, torch.Tensor], prefix: str) -> torch.Tensor:
        """An expert's first weights: its up rows; gated: the gate rows, then the up rows, or, for the clamped unit, the two
        taking turns."""
        if not self.gated:
            return t[prefix + "up"].contiguous()
        if self.glu:
            return torch.stack([t[prefix + "gate"], t[prefix + "up"]], dim=1).flatten(0, 1).contiguous()
        return torch.cat([t[prefix + "gate"], t[prefix + "up"]], dim=0).contiguous()

    def forward(self, x: torch.Tensor, step=None) -> torch.Tensor:
        if self.table_rows:
            s = self._table_sum(x, step)
            out = torch.empty((x.shape[0], self.hidden), dtype=x.dtype, device=x.device)
            weights = torch.full((x.shape[0], self.top), s.scale, dtype=torch.float32, device=x.device)
            ops = kernels.ops()
            ops.moe_combine(out, s.rows, s.place, weights, self.top, add=ops.materialize(s.add) if s.add is not None else None)
            return out
        ops = kernels.ops()
        T, top = x.shape[0], self.top
        idx = torch.empty((T, top), dtype=torch.int32, device=x.device)
        weights = torch.empty((T, top), dtype=torch.float32, device=x.device)
        share = torch.empty((T,), dtype=torch.float32, device=x.device) if self.has_share else None
        ops.router_topk(idx, weights, x, self.w_router, self.softmax, self.renormalize, self.correction, self.groups,
                        self.groups_kept, self.weight_scale, share)
        out = torch.empty((T, self.hidden), dtype=x.dtype, device=x.device)
        if self.identity:
            # the pairs of the experts with tensors are sorted first; the others' output is the token's own row
            offsets, order, place, tiles = ops.moe_align(idx, self.outputs, self.E)
            passing = dict(x=x, pass_from=offsets[self.E:self.E + 1])
        else:
            offsets, order, place, tiles = ops.moe_align(idx, self.E)
            passing = {}
        if self.shared_inter:
            passing.update(add=self._shared(x), share=share)
        if self.E == 0:
            y = torch.empty((T * top, self.hidden), dtype=torch.float32, device=x.device)
        else:
            y = self._experts(x, offsets, order, tiles, weights if self.on_input else None)
        ops.moe_combine(out, y, place, None if self.on_input else weights, top, **passing)
        return out

    def forward_pending(self, x: torch.Tensor, step):
        """With a table: the experts' rows before their sum (the norm that takes them sums them in its own kernel)."""
        return self._table_sum(x, step) if self.table_rows else self.forward(x)

    def _table_sum(self, x: torch.Tensor, step) -> RoutedSum:
        if step is None:
            raise ValueError("routed_mlp: a table of experts needs the step's token ids")
        offsets, order, place, tiles = kernels.ops().moe_align(step.input_ids, self.E, table=self.table)
        y = self._experts(x, offsets, order, tiles, None, getattr(step, "host_ids", None))
        # (after the experts: where its last product is put off, no other may come between it and the sum)
        add = self._shared(x, may_defer=True) if self.shared_inter else None
        return RoutedSum(y, place, self.top, None, 1.0 / self.top, add)

    def _experts(self, x: torch.Tensor, offsets, order, tiles, scale, ids=None) -> torch.Tensor:
        """The experts' outputs, float32 rows sorted by expert; ``scale``: what multiplies their inputs (None: nothing);
        ``ids``: the tokens' ids on the host, with which a table's group sizes need no read-back."""
        ops = kernels.ops()
        T, top = x.shape[0], self.top
        y = torch.empty((T * top, self.hidden), dtype=torch.float32, device=x.device)
        up_width = (2 if self.gated else 1) * self.inter
        if T * top >= self.LIBRARY_ROWS and x.is_cuda and not torch.cuda.is_current_stream_capturing():
            # the experts' input rows in sorted order, weighted and rounded once (the products then read plain rows)
            xs = torch.empty((T * top, self.hidden), dtype=x.dtype, device=x.device)
            ops.moe_gather(xs, x, order, scale, top)
            if self.table_rows and ids is not None:
                counts = np.bincount(self.host_table[ids].reshape(-1), minlength=self.E)
                bounds = [0] + np.cumsum(counts).tolist()
            else:
                bounds = offsets[: self.E + 1].tolist()                  # the one read-back of this path
            a = torch.empty((T * top, up_width), dtype=x.dtype, device=x.device)
            for e in range(self.E):
                lo, hi = bounds[e], bounds[e + 1]
                if hi > lo:
                    ops.linear(a[lo:hi], xs[lo:hi], self.w_up[e])
            a = self._activate(a, bounds[self.E])
            for e in range(self.E):
                lo, hi = bounds[e], bounds[e + 1]
                if hi > lo:
                    ops.linear(y[lo:hi], a[lo:hi], self.w_down[e])
            return y
        a = torch.empty((T * top, self.inter if self.glu else up_width), dtype=x.dtype, device=x.device)
        if self.glu:
            ops.grouped_glu(a, x, self.w_up, order, scale, offsets, tiles, top, self.glu_args)
        elif self.gated:
            # (the first product fetches a pair's token row itself, weighted and rounded as the gather would)
            ops.grouped_linear(a, x, self.w_up, order, scale, offsets, tiles, top)
            a = self._activate(a, T * top)
        else:
            ops.grouped_linear(a, x, self.w_up, order, scale, offsets, tiles, top, self.activation)
        ops.grouped_linear(y, a, self.w_down, None, None, offsets, tiles, 1)
        return y

    def _shared(self, x: torch.Tensor, may_defer: bool = False):
        """The expert that every token uses: down(act(up(x))), or the gated form; ``may_defer``: the last product may be
        put off."""
        ops = kernels.ops()
        T = x.shape[0]
        a = torch.empty((T, self.shared_inter), dtype=x.dtype, device=x.device)
        if self.glu:
            gu = torch.empty((T, 2 * self.shared_inter), dtype=x.dtype, device=x.device)
            ops.glu_pairs(a, ops.linear(gu, x, self.w_shared_up, may_defer=True), self.shared_glu_args)
        elif self.gated:
            gu = torch.empty((T, 2 * self.shared_inter), dtype=x.dtype, device=x.device)
            ops.linear(gu, x, self.w_shared_up)
            ops.silu_mul(a, gu, 0)
        else:
            ops.activation(a, ops.linear(a, x, self.w_shared_up, may_defer=True), self.activation)
        out = torch.empty((T, self.hidden), dtype=x.dtype, device=x.device)
        return ops.linear(out, a, self.w_shared_down, may_defer=may_defer)

    def _activate(self, a: torch.Tensor, rows: int) -> torch.Tensor:
        """The first ``rows`` rows of the experts' first product through the activation (the rows behind them belong
        to experts without tensors and hold nothing); gated experts: act(gate) * up, half as wide."""
        ops = kernels.ops()
        if not self.gated:
            if rows:
                ops.activation(a[:rows], a[:rows], self.activation)
            return a
        g = torch.empty((a.shape[0], self.inter), dtype=a.dtype, device=a.device)
        if rows and self.glu:
            ops.glu_pairs(g[:rows], a[:rows], self.glu_args)
        elif rows:
            ops.silu_mul(g[:rows], a[:rows], 0)
        return g


register("feed_forward", "routed_mlp", RoutedMLP)
