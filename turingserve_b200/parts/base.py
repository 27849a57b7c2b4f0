"""Interfaces of the model's parts and the registries that choose an implementation by
``spec.kind``.

A part knows its own sizes (from its spec) and nothing about the model it sits in.  The model
hands each part its tensors by LOCAL name (e.g. ``q_proj.weight``); which checkpoint prefix those
live under is the architecture's business (``turingserve_b200.config.registry.TensorNames``).

Interfaces
----------
Norm            forward(x, residual=None) -> y          (residual updated in place when given; x may be a
                                                         product left unreduced by its kernel, which a
                                                         norm either passes to a kernel that finishes it
                                                         or turns into a tensor with ops().materialize)
PositionEncoding  tables()/apply are private to the mixers that accept it
Mixer           forward(x, step, cache, state) -> y     cache_need() / state_need() declare memory
FeedForward     forward(x) -> y                         (forward(x, step) where ``wants_step``; mixers and feed-forwards get tensors; they may
                                                         return what ops().linear(..., may_defer=True) gave)
Block           forward(h, residual, step, cache, state) -> (h, residual)   (h is whatever the arrangement's own
                                                         norm takes: a tensor, a product put off, a ``BranchSum``)

``step`` is a ``StepInputs`` (turingserve_b200.engine.batch): the flat batch on the device.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable

import torch


@dataclass(frozen=True)
class ParamSpec:
    """One checkpoint tensor a part reads.

    ``compute_dtype`` True: converted to the engine's dtype (operands of matrix products,
    embeddings).  False: a tensor stored in 32 bits stays in 32 bits, anything else is converted.
    ``integer`` True: an integer table, kept as int32.
    A dimension None is whatever the checkpoint has (the part reads it from the tensor it gets); the random-weights mode
    makes it ``free`` long.
    """

    shape: tuple[int | None, ...]
    compute_dtype: bool = True
    integer: bool = False
    # how the random-weights mode fills it: "normal" | "ones" | "zeros" | "identity"; an integer table: "zeros", or
    # "distinct": every row so many different numbers below ``high``
    init: str = "normal"
    high: int = 0
    free: int = 0

    def fits(self, shape) -> bool:
        return len(shape) == len(self.shape) and all(n is None or n == got for n, got in zip(self.shape, shape))

    @property
    def sizes(self) -> tuple[int, ...]:
        """The shape the random-weights mode gives it."""
        return tuple(self.free if n is None else n for n in self.shape)


@dataclass(frozen=True)
class CacheNeed:
    """What a mixer wants from the paged cache: keys and values of ``num_kv_heads`` x ``head_dim``
    per token; ``window`` None keeps every token, an integer keeps the last ``window`` of them (and the first ``keep_first``).
    ``value_dim``: the width of a value row where it differs from a key row's ``head_dim`` (the
    group's keys and values are then two tensors instead of one pool).  ``chunk`` c: a position sees only
    the keys of its own block of c positions (blocks counted from position 0), so tokens before the block of
    the next position need not be kept."""

    num_kv_heads: int
    head_dim: int
    window: int | None = None
    value_dim: int | None = None
    chunk: int | None = None
    keep_first: int = 0             # with a window: the first so many tokens stay visible, so they are kept too

    @property
    def v_dim(self) -> int:
        return self.head_dim if self.value_dim is None else self.value_dim


@dataclass(frozen=True)
class StateNeed:
    """Fixed-size per-request state of a mixer (zeroed when a request is admitted)."""

    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32


class Part:
    """Base of all parts: declares parameters, receives them."""

    def parameters(self) -> dict[str, ParamSpec]:
        return {}

    def load(self, tensors: dict[str, torch.Tensor]) -> None:
        """Receive the tensors named by ``parameters()``, already on the device and converted."""
        if tensors:
            raise ValueError(f"{type(self).__name__} takes no tensors, got {sorted(tensors)}")


class Norm(Part):
    def forward(self, x: torch.Tensor, residual: torch.Tensor | None = None) -> torch.Tensor:
        raise NotImplementedError


class Mixer(Part):
    def cache_need(self) -> CacheNeed | None:
        return None

    def state_need(self) -> StateNeed | None:
        return None

    def forward(self, x: torch.Tensor, step, cache, state: torch.Tensor | None) -> torch.Tensor:
        raise NotImplementedError

    # A mixer of the form  W_out f(W_in x + b)  may expose its two products, so that a mixer made of several
    # (``parts.paired_mixer``) runs ONE input product and ONE output product for all of them:
    #   in_projection()  -> (weight [n_in, hidden], bias [n_in] or None), after load()
    #   out_projection() -> weight [hidden, n_heads]
    #   heads_forward(proj [T, n_in], step, cache, state, out [T, n_heads], scale): out = scale * f(proj); ``proj`` and
    #   ``out`` are column slices of wider tensors (rows not contiguous).
    def in_projection(self):
        raise NotImplementedError(f"{type(self).__name__} does not expose its projections")

    def out_projection(self):
        raise NotImplementedError(f"{type(self).__name__} does not expose its projections")

    def heads_forward(self, proj, step, cache, state, out, scale: float = 1.0) -> None:
        raise NotImplementedError(f"{type(self).__name__} does not expose its projections")


class FeedForward(Part):
    # whether ``forward`` also wants the step (a feed-forward that looks at the tokens' ids); the block then calls
    # forward(x, step)
    wants_step = False

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError

    def forward_pending(self, x: torch.Tensor, step):
        """The output as a norm that finishes sums may take it: what ``forward`` gives, or a ``RoutedSum``."""
        return self.forward(x, step) if self.wants_step else self.forward(x)


@dataclass
class BranchSum:
    """What a layer whose branches all read one norm's output leaves pending: the branches' outputs (``second``
    may be None) and the constant their sum is multiplied by on its way into the residual stream.  The norm that
    follows takes them into the stream in its own kernel.  An embedding on its way into a stream that is about
    to start has the same form (the rows and their multiplier)."""

    first: Any
    second: Any = None
    scale: float = 1.0


@dataclass
class RoutedSum:
    """What a routed feed-forward leaves before its last kernel: the experts' output rows (float32, sorted by expert), the
    sorted place of every (token, choice) pair, the weights (one per pair, or None) and a constant, and the output of an
    expert that every token uses (``add``: a tensor, a product put off or None).  Valid until the next routed feed-forward
    runs (``place`` is a work buffer of the kernels)."""

    rows: torch.Tensor
    place: torch.Tensor
    top: int
    pair_weights: Any = None
    scale: float = 1.0
    add: Any = None


@dataclass
class NormedUpdate:
    """What a sublayer whose OUTPUT is normed leaves pending: the output ``y`` (a tensor, a product put off or a
    ``RoutedSum``) and the norm (``parts.rmsnorm.PostRMSNorm``) through which it enters the stream.  ``base``: the rows the
    stream starts from (where this is the model's first update)."""

    y: Any
    norm: Any
    base: Any = None


@dataclass
class StreamUpdate:
    """What a sublayer on a residual stream of several copies leaves pending: its output ``y`` (a tensor or a product
    put off) and the link (``parts.stream_link.StreamLink``: the mix matrix and the output weights) by which it comes
    back into the copies.  The norm that follows carries the write-back out in its own kernel."""

    y: Any
    link: Any


@dataclass(frozen=True)
class BuildContext:
    """What every part constructor gets besides its spec."""

    hidden_size: int
    dtype: torch.dtype
    device: torch.device
    max_positions: int              # longest sequence the engine will run (sizes position tables)


_REGISTRIES: dict[str, dict[str, Callable[[Any, BuildContext], Any]]] = {
    "norm": {}, "position": {}, "mixer": {}, "feed_forward": {}, "block": {}, "link": {},
}


def register(family: str, kind: str, factory: Callable[[Any, BuildContext], Any]) -> None:
    """Register ``factory(spec, ctx) -> part`` for ``spec.kind == kind`` in ``family``
    (norm | position | mixer | feed_forward | block | link)."""
    _REGISTRIES[family][kind] = factory


def build(family: str, spec: Any, ctx: BuildContext):
    _load_builtin()
    kind = spec if isinstance(spec, str) else getattr(spec, "kind", None)
    try:
        factory = _REGISTRIES[family][kind]
    except KeyError:
        known = ", ".join(sorted(_REGISTRIES[family])) or "none"
        raise ValueError(f"no {family} registered for kind {kind!r} (registered: {known})") from None
    return factory(spec, ctx)


_loaded = False


def _load_builtin() -> None:
    global _loaded
    if not _loaded:
        _loaded = True
        from turingserve_b200.parts import (  # noqa: F401
            attention, block, capped_attention, delta_rule, diff_attention, gated_mlp, latent_attention, lightning, mamba2,
            mlp, normed_attention, paired_mixer, rglru, rmsnorm, rotary, routed_mlp, sink_attention, stream_link, wkv)


def build_block(layer_spec: Any, ctx: BuildContext):
    """Build one layer; ``layer_spec.arrangement`` chooses the wiring."""
    _load_builtin()
    try:
        factory = _REGISTRIES["block"][layer_spec.arrangement]
    except KeyError:
        known = ", ".join(sorted(_REGISTRIES["block"])) or "none"
        raise ValueError(f"no block arrangement {layer_spec.arrangement!r} (registered: {known})") from None
    return factory(layer_spec, ctx)
