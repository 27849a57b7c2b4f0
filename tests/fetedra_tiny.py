"""Tiny Fetedra configurations of the test-suite and their random weights.  They differ in every size and option: width,
vocabulary (no multiples of anything), eps, 1 to 3 copies of the stream and none, the order of the two mixers, layers without a
feed-forward (the first layer too), heads of 7 to 64 channels, ranks of the decay from 5 to 32, latents and head parts that all
differ, rotation over part of the rotated part and all of it, windows of 1 to 70 positions and none, experts with top 1 and more,
groups of which one, some and all are kept (groups of one expert too), scales of the weights, with and without a shared expert;
clamped early, late and hardly; logit scales; page size."""

from __future__ import annotations

import json
import os

import numpy as np
import torch
from safetensors.torch import save_file

from turingserve_b200.models.fetedra import make_config
from turingserve_b200.weights.random_init import random_tensors


def wkv(heads, dim, rank):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "decay_rank": rank}}


def lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, window=None, rot=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim if rot is None else rot}}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, groups=(1, 1), scale=1.0, shared=None):
    """groups: (count, keep); shared: (ff, limit)."""
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit},
         "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups[0], "keep": groups[1]}}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


# name -> (config arguments, seed, cache page size)
TINY = {
    # sizes that are no multiples of 8; three copies; a window shorter than a page and one that crosses pages
    "A": (dict(width=60, vocab=131, eps=1e-5, streams=3, logit_scale=0.7, layers=[
        {**lat(3, 10, 6, 12, 20, 28, 0.4, 100.0, 7), "mlp": moe(12, 3, 20, 0.6, (4, 2), 1.7, (28, 0.9))},
        {**wkv(3, 20, 12), "mlp": dense(52)},
        {**lat(5, 6, 10, 8, 14, 18, 0.5, 40.0, 21, 6), "mlp": None},
        {**wkv(2, 7, 5), "mlp": moe(6, 2, 12, 1.5, (6, 3), 0.8)},
    ]), 71, 16),
    # a time mixer without a feed-forward first; one copy with a link of its own; top 1; no groups; one group kept of three; pages
    # of 8; a window of 40, and none
    "B": (dict(width=48, vocab=257, eps=1e-6, streams=1, logit_scale=1.3, layers=[
        {**wkv(4, 16, 8), "mlp": None},
        {**wkv(1, 40, 24), "mlp": moe(9, 1, 16, 0.8, (3, 1), 1.4, (12, 0.5))},
        {**lat(4, 12, 8, 10, 24, 16, 0.4, 500.0, 40), "mlp": moe(5, 2, 24, 1.0, (1, 1), 2.2)},
        {**lat(2, 8, 4, 20, 8, 24, 0.6, 30.0), "mlp": dense(36)},
    ]), 72, 8),
    # multiples of 64, pages of 64: the tensor-core products of few rows, the one-kernel steps, cached rows of 320 with values
    # of 256 (the tensor-core attention in bfloat16) behind a window of 70 and none
    "C": (dict(width=128, vocab=300, eps=1e-6, streams=2, logit_scale=0.4, layers=[
        {**wkv(2, 64, 32), "mlp": dense(192)},
        {**lat(3, 32, 64, 40, 64, 256, 0.12, 10000.0, 70), "mlp": moe(8, 2, 64, 0.7, (2, 1), 2.5, (32, 0.6))},
        {**wkv(4, 32, 16), "mlp": moe(16, 4, 32, 0.8, (8, 4), 1.1, (64, 0.9))},
        {**lat(6, 64, 64, 32, 96, 256, 0.1, 300000.0), "mlp": None},
    ]), 73, 64),
    # the ordinary residual sum (no streams in the configuration); a position that sees itself alone; two experts
    "D": (dict(width=32, vocab=50, eps=1e-5, layers=[
        {**lat(2, 8, 6, 12, 10, 14, 0.5, 30.0, 1), "mlp": moe(2, 2, 16, 0.5, (2, 2), 0.6, (12, 0.7))},
        {**wkv(2, 12, 9), "mlp": dense(24)},
    ]), 74, 16),
}

# how much larger than the base deviation a tensor's entries are (by the end of its name)
BOOST = {"embed": 12.0, ".gate": 4.0, ".up": 4.0, ".down": 2.0, ".router": 6.0, ".sg": 8.0, "mix.g": 4.0, "mix.r": 3.0, "mix.k": 3.0,
         "mix.v": 3.0, ".w1": 6.0, ".w2": 8.0, ".uq": 4.0, ".dq": 3.0, ".dkv": 3.0, ".uk": 4.0, ".uv": 3.0, "mix.o": 2.0}


def tiny_config(name: str):
    return make_config(**TINY[name][0])


def page_size(name: str) -> int:
    return TINY[name][2]


def tiny_tensors(cfg, seed: int, std: float = 0.05) -> dict[str, torch.Tensor]:
    tensors = random_tensors(cfg, seed, std)
    g = torch.Generator().manual_seed(seed + 1000)
    rnd = lambda t, s: s * torch.randn(t.shape, generator=g)
    for n, t in tensors.items():
        if n.endswith((".norm1", ".norm2")) or n == "final.norm":     # stored around zero: the scale is 1 + w
            new = rnd(t, 0.3)
        elif n.endswith(".norm"):                    # the latents' and the heads' norms: plain scales around one
            new = 1.0 + rnd(t, 0.3)
        elif ".mu." in n:
            new = 0.5 + rnd(t, 0.3)
        elif n.endswith(".w0"):                      # memories from a token to hundreds
            new = 1.0 - 7.0 * torch.rand(t.shape, generator=g)
        elif n.endswith(".u"):
            new = rnd(t, 0.7)
        elif n.endswith(".sink"):
            new = rnd(t, 1.0)
        elif n.endswith(".correction"):              # some choice scores are negative
            new = -0.5 + rnd(t, 0.2)
        elif n.endswith((".in", ".out")):
            new = 0.7 + rnd(t, 0.3)
        elif n.endswith("hc1.mix") or n.endswith("hc2.mix"):
            new = 0.9 * torch.eye(t.shape[0]) + rnd(t, 0.15)
        else:
            new = t.float()
            for end, f in BOOST.items():
                if n.endswith(end):
                    new = new * f
        tensors[n] = new.to(t.dtype)
    return tensors


def make_tiny_folder(name: str, base, std: float = 0.05) -> str:
    kw, seed, _ = TINY[name]
    folder = os.path.join(str(base), f"fetedra_{name}")
    if os.path.exists(os.path.join(folder, "model.safetensors")):
        return folder
    cfg = make_config(**kw)
    from turingserve_b200.config.registry import get_architecture
    os.makedirs(folder, exist_ok=True)
    c = get_architecture("Fetedra").to_config_json(cfg)
    for entry in c["layers"]:
        entry["mixer"].pop("decay_rank", None)       # (the tensors say it)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as f:
        json.dump(c, f)
    save_file(tiny_tensors(cfg, seed, std), os.path.join(folder, "model.safetensors"))
    return folder


def random_ids(n: int, vocab: int, seed: int) -> list[int]:
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()
