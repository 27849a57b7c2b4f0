"""Suranex: config.json keys -> ``ModelConfig``, checkpoint tensor names, and the model class.

A decoder whose layers are, in the order the configuration lists them, one of two mixers and a feed-forward or none,
over a residual stream in 32-bit, with norms on the sublayers' OUTPUTS only: x <- x + norm1(mixer(x)), x <- x +
norm2(ff(x)); the sublayers read x itself.  Norms are RMS norms whose weights are stored around zero (scale 1 + w).
``attention``: grouped-query softmax attention with learned norms on the heads of q and k before their rotation (pairs of
halves, YaRN-blended frequencies), values over their root mean square and turned by their positions (the heads' outputs
turned back), capped scores, a window behind which the first tokens stay visible, and a sigmoid gate per head.
``rglru``: the recurrent block of a real-gated linear recurrent unit.  Feed-forward: experts g sigmoid(1.702 g) (u + 1)
with clamped g and u, chosen by a table of token ids with equal weights, and a shared expert of the same form.  The output
head has a matrix of its own behind the model's norm.  Every size and constant comes from config.json but for the
numbers the design fixes: the recurrence's 8, the gated unit's 1.702 and 1, and the halves' pairing.
"""

from __future__ import annotations

import torch

from turingserve_b200.config.model_config import (
    LayerRun, LayerSpec, ModelConfig, NormedAttentionSpec, PostRMSNormSpec, RGLRUSpec, RoutedMLPSpec, YarnRotarySpec)
from turingserve_b200.config.registry import (
    Architecture, LayerTensorNames, TensorNames, register_architecture)
from turingserve_b200.parts.base import NormedUpdate
from turingserve_b200.parts.model import DecoderModel

NAME = "Suranex"
# the rotation's angles are computed from the position itself: nothing in the design bounds a sequence
NO_POSITION_LIMIT = 1 << 30
NO_LIMIT = float("inf")


def _require(c: dict, key: str, where: str = "config.json"):
    if key not in c:
        raise ValueError(f"{where} is missing required key {key!r}")
    return c[key]


def _rotation(rot: dict, where: str):
    if int(rot.get("dims", 0)) <= 0:
        return None
    kw = {}
    sc = rot.get("scaling") or None
    if sc:
        kw = dict(factor=float(_require(sc, "factor", where)), original=float(_require(sc, "original", where)),
                  fast=float(_require(sc, "fast", where)), slow=float(_require(sc, "slow", where)))
    return YarnRotarySpec(base=float(_require(rot, "base", where)), dims=int(rot["dims"]), pairing="halves", **kw)


def _mixer(kind: str, m: dict, eps: float, where: str):
    if kind == "attention":
        heads, dim = int(_require(m, "heads", where)), int(_require(m, "dim", where))
        rot, mask, cap = m.get("rot") or None, m.get("mask") or None, m.get("softcap")
        return NormedAttentionSpec(
            num_heads=heads, num_kv_heads=int(m.get("kv_heads", heads)), key_dim=dim, value_dim=int(m.get("vdim", dim)),
            scale=float(_require(m, "scale", where)), norm_eps=eps, position=_rotation(rot, where) if rot else None,
            softcap=float(cap) if cap else None, window=int(_require(mask, "size", where)) if mask else None,
            keep_first=int(mask.get("keep_first", 0)) if mask else 0,
            value_base=float(_require(rot, "base", where)) if rot else None)
    if kind == "rglru":
        return RGLRUSpec(width=int(_require(m, "width", where)), num_blocks=int(_require(m, "blocks", where)),
                         conv_taps=int(_require(m, "conv", where)))
    raise ValueError(f"{where}: unknown layer type {kind!r} (known: attention, rglru)")


def _feed_forward(f: dict | None, vocab: int, where: str):
    if f is None:
        return None
    kind = _require(f, "kind", where)
    if kind != "moe":
        raise ValueError(f"{where}: unknown feed-forward kind {kind!r} (known: moe)")
    router, expert, shared = _require(f, "router", where), _require(f, "expert", where), f.get("shared") or None
    limit = lambda e: NO_LIMIT if e.get("limit") is None else float(e["limit"])
    kw = dict(shared_intermediate_size=int(_require(shared, "ff", where)), shared_glu_limit=limit(shared)) if shared else {}
    return RoutedMLPSpec(
        num_experts=int(_require(router, "experts", where)), top_k=int(_require(router, "top", where)),
        intermediate_size=int(_require(expert, "ff", where)), activation="clamped_glu", weight_on="output", gated=True,
        table_rows=vocab, glu_limit=limit(expert), **kw)


def parse_config(c: dict, gen: dict | None = None) -> ModelConfig:
    eps = float(_require(_require(c, "norm"), "eps", "norm"))
    vocab = int(_require(c, "vocab"))
    norm = PostRMSNormSpec(eps=eps, weight_offset=1.0, weight_name="")
    layers = []
    for i, entry in enumerate(_require(c, "layers")):
        where = f"layers[{i}]"
        roles = dict(mixer=_mixer(_require(entry, "type", where), _require(entry, "mixer", where), eps, where), mixer_norm=norm)
        ff = _feed_forward(entry.get("mlp"), vocab, where)
        if ff is not None:
            roles.update(feed_forward=ff, ffn_norm=norm)
        layers.append(LayerSpec("post_norm_stream", **roles))
    eos = (gen or {}).get("eos_token_id", c.get("eos_token_id"))
    eos_ids = () if eos is None else ((int(eos),) if isinstance(eos, int) else tuple(int(x) for x in eos))
    return ModelConfig(
        architecture=NAME, hidden_size=int(_require(c, "width")), vocab_size=vocab, layers=tuple(layers),
        schedule=tuple(LayerRun(i) for i in range(len(layers))), final_norm=norm, tie_word_embeddings=False,
        max_position_embeddings=int(c.get("max_positions", NO_POSITION_LIMIT)), eos_token_ids=eos_ids,
        bos_token_id=c.get("bos_token_id"))


def tensor_names(cfg: ModelConfig) -> TensorNames:
    """'l<i>.norm1', 'l<i>.mix.<name>', 'l<i>.norm2', 'l<i>.mlp.<name>'; 'embed', 'final.norm', 'head'.  A norm's weight is
    named by the prefix itself."""
    layers = []
    for i, spec in enumerate(cfg.layers):
        names = dict(mixer=f"l{i}.mix.", mixer_norm=f"l{i}.norm1")
        if "feed_forward" in spec.roles:
            names.update(feed_forward=f"l{i}.mlp.", ffn_norm=f"l{i}.norm2")
        layers.append(LayerTensorNames(**names))
    return TensorNames(embedding="embed", lm_head="head", final_norm="final.norm", layers=tuple(layers))


def _entry(spec: LayerSpec) -> dict:
    m = spec.mixer
    if isinstance(m, RGLRUSpec):
        entry = {"type": "rglru", "mixer": {"width": m.width, "blocks": m.num_blocks, "conv": m.conv_taps}}
    else:
        mixer = {"heads": m.num_heads, "kv_heads": m.num_kv_heads, "dim": m.key_dim, "vdim": m.value_dim, "scale": m.scale}
        if m.value_base is not None:
            mixer["rot"] = {"base": m.value_base, "dims": m.position.dims if m.position is not None else 0}
            if m.position is not None and m.position.factor:
                r = m.position
                mixer["rot"]["scaling"] = {"factor": r.factor, "original": r.original, "fast": r.fast, "slow": r.slow}
        if m.softcap:
            mixer["softcap"] = m.softcap
        if m.window:
            mixer["mask"] = {"size": m.window, "keep_first": m.keep_first}
        entry = {"type": "attention", "mixer": mixer}
    f = spec.roles.get("feed_forward")
    if f is None:
        entry["mlp"] = None
        return entry

    def sized(ff: int, limit: float) -> dict:
        return {"ff": ff} if limit == NO_LIMIT else {"ff": ff, "limit": limit}
    entry["mlp"] = {"kind": "moe", "expert": sized(f.intermediate_size, f.glu_limit),
                    "router": {"experts": f.num_experts, "top": f.top_k}}
    if f.shared_intermediate_size:
        entry["mlp"]["shared"] = sized(f.shared_intermediate_size, f.shared_glu_limit)
    return entry


def to_config_json(cfg: ModelConfig) -> dict:
    out = {"architecture": NAME, "width": cfg.hidden_size, "vocab": cfg.vocab_size,
           "layers": [_entry(cfg.run_layer(r)) for r in range(cfg.num_runs)], "norm": {"eps": cfg.final_norm.eps}}
    if cfg.max_position_embeddings != NO_POSITION_LIMIT:
        out["max_positions"] = cfg.max_position_embeddings
    if cfg.eos_token_ids:
        out["eos_token_id"] = list(cfg.eos_token_ids) if len(cfg.eos_token_ids) > 1 else cfg.eos_token_ids[0]
    return out


def make_config(*, width: int, vocab: int, layers: list[dict], eps: float = 1e-6, eos_token_id: int | None = None) -> ModelConfig:
    """A Suranex ``ModelConfig`` from sizes (through the same parser as config.json); ``layers`` as the configuration
    file lists them."""
    c = {"architecture": NAME, "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}}
    if eos_token_id is not None:
        c["eos_token_id"] = eos_token_id
    return parse_config(c)


class SuranexModel(DecoderModel):
    """The decoder whose last layer's output norm, its add to the stream and the model's own norm are one kernel."""

    def finish(self, h, residual):
        if not isinstance(h, NormedUpdate):
            raise TypeError(f"suranex: the last layer leaves a NormedUpdate, not {type(h).__name__}")
        return h.norm.forward(h.y, residual, base=h.base, reader=self.final_norm)


register_architecture(Architecture(NAME, parse_config, tensor_names, to_config_json, build_model=SuranexModel))
