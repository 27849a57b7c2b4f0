"""Fetedra: config.json keys -> ``ModelConfig``, and checkpoint tensor names.

A decoder whose layers are, in the order the configuration lists them, one of two mixers and a feed-forward or none,
pre-norm over a residual stream in 32-bit kept as several copies (``streams``: hyper-connections, every sublayer with a read
vector, a write vector and a mix matrix of its own; without the key the ordinary residual sum).  ``wkv``: a matrix state per
head that fades channel by channel at rates the token chooses, over mixes of a token's input with its predecessor's.
``latent_attention``: attention through low-rank latents with a rotated part (pairs of halves), a sliding window, a learned
sink per head in the softmax's denominator and a gate per head.  Feed-forwards: dense gated with SiLU, or routed: sigmoid
scores, a correction that enters the choice only, groups of neighbouring experts of which the best are kept, weights
renormalised times a constant, experts that are clamped gated units (slope 1.702, offset 1) with a limit from the configuration,
plus a gated shared expert of the same form with a size and limit of its own.  Norms are RMS norms whose weights are stored
around zero (scale 1 + w).  The output head is the embedding table itself after the model's norm, times ``logit_scale``.
Every size and constant comes from config.json, but for the rank of the decay's products, which the tensors give.
"""

from __future__ import annotations

from turingserve_b200.config.model_config import (
    GatedMLPSpec, HalfRotarySpec, HyperRMSNormSpec, LatentAttentionSpec, LayerRun, LayerSpec, ModelConfig, RoutedMLPSpec,
    StreamLinkSpec, WKVSpec)
from turingserve_b200.config.registry import (
    Architecture, LayerTensorNames, TensorNames, register_architecture)
from turingserve_b200.parts.model import HyperStreamModel

NAME = "Fetedra"
# the rotation's angles are computed from the position itself: nothing in the design bounds a sequence
NO_POSITION_LIMIT = 1 << 30
FF_NAMES = ("gate", "up", "down")
GLU_SLOPE, GLU_OFFSET = 1.702, 1.0


def _require(c: dict, key: str, where: str = "config.json"):
    if key not in c:
        raise ValueError(f"{where} is missing required key {key!r}")
    return c[key]


def _mixer(kind: str, m: dict, eps: float, where: str):
    heads, dim = int(_require(m, "heads", where)), int(_require(m, "dim", where))
    if kind == "wkv":
        rank = m.get("decay_rank")
        return WKVSpec(num_heads=heads, head_dim=dim, norm_eps=eps, decay_rank=None if rank is None else int(rank))
    if kind == "latent_attention":
        rope_dim = int(_require(m, "rot_dim", where))
        rot = _require(m, "rot", where)
        dims = int(rot.get("dims", rope_dim))
        if dims > rope_dim or dims % 2:
            raise ValueError(f"{where}: rot.dims {dims} must be even and at most rot_dim {rope_dim}")
        mask = m.get("mask")
        return LatentAttentionSpec(
            num_heads=heads, nope_dim=dim, rope_dim=rope_dim, value_dim=int(_require(m, "vdim", where)),
            q_rank=int(_require(m, "q_rank", where)), kv_rank=int(_require(m, "kv_rank", where)),
            scale=float(_require(m, "scale", where)), norm_eps=eps,
            position=HalfRotarySpec(base=float(_require(rot, "base", where)), dims=dims),
            window=int(_require(mask, "size", where)) if mask is not None else None, sinks=True, head_gate=True)
    raise ValueError(f"{where}: unknown layer type {kind!r} (known: wkv, latent_attention)")


def _feed_forward(f: dict | None, where: str):
    if f is None:
        return None
    kind = _require(f, "kind", where)
    if kind == "dense":
        return GatedMLPSpec(intermediate_size=int(_require(f, "ff", where)), activation="silu", names=FF_NAMES)
    if kind == "moe":
        router, expert = _require(f, "router", where), _require(f, "expert", where)
        shared, groups = f.get("shared") or None, router.get("groups") or {"count": 1, "keep": 1}
        kw = {}
        if shared:
            kw = dict(shared_intermediate_size=int(_require(shared, "ff", where)), shared_gate=True,
                      shared_glu_limit=float(_require(shared, "limit", where)))
        return RoutedMLPSpec(
            num_experts=int(_require(router, "experts", where)), top_k=int(_require(router, "top", where)),
            intermediate_size=int(_require(expert, "ff", where)), activation="clamped_glu", gated=True, scoring="sigmoid",
            renormalize=True, weight_on="output", correction=True, groups=int(_require(groups, "count", where)),
            groups_kept=int(_require(groups, "keep", where)), weight_scale=float(router.get("scale", 1.0)),
            glu_limit=float(_require(expert, "limit", where)), glu_slope=GLU_SLOPE, glu_offset=GLU_OFFSET, **kw)
    raise ValueError(f"{where}: unknown feed-forward kind {kind!r} (known: dense, moe)")


def parse_config(c: dict, gen: dict | None = None) -> ModelConfig:
    eps = float(_require(_require(c, "norm"), "eps", "norm"))
    streams = c.get("streams")
    S = int(streams) if streams is not None else 1
    if S < 1:
        raise ValueError(f"streams = {S}")
    norm = HyperRMSNormSpec(eps=eps, streams=S, weight_offset=1.0, weight_name="")
    link = StreamLinkSpec(streams=S, learned=streams is not None)
    layers = []
    for i, entry in enumerate(_require(c, "layers")):
        where = f"layers[{i}]"
        mixer = _mixer(_require(entry, "type", where), _require(entry, "mixer", where), eps, where)
        ff = _feed_forward(entry.get("mlp"), where)
        roles = dict(mixer=mixer, mixer_norm=norm, mixer_link=link)
        if ff is not None:
            roles.update(feed_forward=ff, ffn_norm=norm, ffn_link=link)
        layers.append(LayerSpec("hyper_streams", **roles))
    eos = (gen or {}).get("eos_token_id", c.get("eos_token_id"))
    eos_ids = () if eos is None else ((int(eos),) if isinstance(eos, int) else tuple(int(x) for x in eos))
    extras = (("logit_scale", float(c.get("logit_scale", 1.0))), ("streams", None if streams is None else S))
    return ModelConfig(
        architecture=NAME, hidden_size=int(_require(c, "width")), vocab_size=int(_require(c, "vocab")),
        layers=tuple(layers), schedule=tuple(LayerRun(i) for i in range(len(layers))), final_norm=norm, tie_word_embeddings=True,
        max_position_embeddings=int(c.get("max_positions", NO_POSITION_LIMIT)), eos_token_ids=eos_ids,
        bos_token_id=c.get("bos_token_id"), extras=extras)


def tensor_names(cfg: ModelConfig) -> TensorNames:
    """'l<i>.norm1', 'l<i>.mix.<name>', 'l<i>.hc1.<name>', 'l<i>.norm2', 'l<i>.mlp.<name>', 'l<i>.hc2.<name>'; 'embed',
    'final.norm'.  A norm's weight is named by the prefix itself."""
    layers = []
    for i, spec in enumerate(cfg.layers):
        names = dict(mixer=f"l{i}.mix.", mixer_norm=f"l{i}.norm1", mixer_link=f"l{i}.hc1.")
        if "feed_forward" in spec.roles:
            names.update(feed_forward=f"l{i}.mlp.", ffn_norm=f"l{i}.norm2", ffn_link=f"l{i}.hc2.")
        layers.append(LayerTensorNames(**names))
    return TensorNames(embedding="embed", lm_head="embed", final_norm="final.norm", layers=tuple(layers))


def _entry(spec: LayerSpec) -> dict:
    m = spec.mixer
    if isinstance(m, WKVSpec):
        entry = {"type": "wkv", "mixer": {"heads": m.num_heads, "dim": m.head_dim}}
        if m.decay_rank is not None:
            entry["mixer"]["decay_rank"] = m.decay_rank
    else:
        entry = {"type": "latent_attention",
                 "mixer": {"heads": m.num_heads, "dim": m.nope_dim, "rot_dim": m.rope_dim, "vdim": m.value_dim,
                           "q_rank": m.q_rank, "kv_rank": m.kv_rank, "scale": m.scale,
                           "rot": {"base": m.position.base, "dims": m.position.dims}}}
        if m.window:
            entry["mixer"]["mask"] = {"size": m.window}
    f = spec.roles.get("feed_forward")
    if f is None:
        entry["mlp"] = None
    elif isinstance(f, GatedMLPSpec):
        entry["mlp"] = {"kind": "dense", "ff": f.intermediate_size}
    else:
        entry["mlp"] = {"kind": "moe", "expert": {"ff": f.intermediate_size, "limit": f.glu_limit},
                        "router": {"experts": f.num_experts, "top": f.top_k, "scale": f.weight_scale,
                                   "groups": {"count": f.groups, "keep": f.groups_kept}}}
        if f.shared_intermediate_size:
            entry["mlp"]["shared"] = {"ff": f.shared_intermediate_size, "limit": f.shared_glu_limit}
    return entry


def to_config_json(cfg: ModelConfig) -> dict:
    out = {"architecture": NAME, "width": cfg.hidden_size, "vocab": cfg.vocab_size,
           "layers": [_entry(cfg.layers[run.layer]) for run in cfg.schedule], "norm": {"eps": cfg.final_norm.eps},
           "logit_scale": cfg.extra("logit_scale", 1.0)}
    if cfg.extra("streams") is not None:
        out["streams"] = cfg.extra("streams")
    if cfg.max_position_embeddings != NO_POSITION_LIMIT:
        out["max_positions"] = cfg.max_position_embeddings
    if cfg.eos_token_ids:
        out["eos_token_id"] = list(cfg.eos_token_ids) if len(cfg.eos_token_ids) > 1 else cfg.eos_token_ids[0]
    return out


def make_config(*, width: int, vocab: int, layers: list[dict], eps: float = 1e-6, streams: int | None = None,
                logit_scale: float = 1.0, eos_token_id: int | None = None) -> ModelConfig:
    """A Fetedra ``ModelConfig`` from sizes (through the same parser as config.json); ``layers`` as the configuration file
    lists them."""
    c = {"architecture": NAME, "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps},
         "logit_scale": logit_scale}
    if streams is not None:
        c["streams"] = streams
    if eos_token_id is not None:
        c["eos_token_id"] = eos_token_id
    return parse_config(c)


register_architecture(Architecture(NAME, parse_config, tensor_names, to_config_json, build_model=HyperStreamModel))
