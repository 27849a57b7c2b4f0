"""Tiny Suranex configurations of the test-suite and their random weights.  They differ in every size and option: width,
vocabulary (no multiples of anything), eps, the order of the two mixers, layers without a feed-forward (the first layer
too), heads and kv heads, key and value widths that differ, rotation over part of a head, all of it and none, frequencies
blended and plain, caps and none, windows of 1 to 40 positions that keep 0 to 70 first tokens, no window; recurrent units
of 1 to 8 parts (1 to 64 channels each) with filters of 1 to 4 taps; experts with top 1 and top = all, with and without a
shared expert, clamped early, late and not at all; page size."""

from __future__ import annotations

import json
import os

import numpy as np
import torch
from safetensors.torch import save_file

from turingserve_b200.models.suranex import make_config
from turingserve_b200.weights.random_init import random_tensors


def att(heads, kv, dim, vdim, scale, rot=None, mask=None, cap=None):
    """rot: (base, dims[, (factor, original, fast, slow)]); mask: (size, keep_first)."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    if mask:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]}
    if cap:
        m["softcap"] = cap
    return {"type": "attention", "mixer": m}


def rec(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def moe(experts, top, ff, limit=None, shared=None):
    """shared: (ff, limit)."""
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if limit is not None:
        m["expert"]["limit"] = limit
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


# name -> (config arguments, seed, cache page size)
TINY = {
    # a window of 7 that keeps 3 first tokens (inside the first page) and one of 21 that keeps 18 (past a page's edge);
    # frequencies that stay, blend and slow; parts of 20 channels, a filter of 4 taps
    "A": (dict(width=72, vocab=131, eps=1e-5, layers=[
        {**att(4, 2, 16, 8, 0.4, (100.0, 8, (8.0, 40.0, 4.0, 1.0)), (7, 3), 5.0), "mlp": moe(5, 2, 24, 0.8, (16, 0.5))},
        {**rec(60, 3, 4), "mlp": moe(5, 2, 24, 0.6, (40, 1.1))},
        {**att(3, 1, 10, 14, 0.5, (50.0, 10), (21, 18)), "mlp": None},
        {**rec(48, 2, 2), "mlp": moe(4, 4, 8, 1.5)},
    ]), 61, 16),
    # a recurrent layer without a feed-forward first; one part, one tap (no memory of the filter); a window that keeps
    # nothing, and none; six heads on one kv head, five on five; top 1; no shared expert; experts never clamped; pages of 8
    "B": (dict(width=48, vocab=257, eps=1e-6, layers=[
        {**rec(36, 1, 1), "mlp": None},
        {**att(6, 1, 12, 20, 0.45, (500.0, 4), (40, 0)), "mlp": moe(6, 1, 20)},
        {**att(5, 5, 10, 6, 0.45, None, None, 3.0), "mlp": None},
        {**rec(64, 8, 3), "mlp": moe(3, 3, 28, 0.7, (24, 0.9))},
        {**att(2, 2, 8, 8, 0.6, (30.0, 8)), "mlp": moe(7, 2, 16, 1.0, (8, 0.4))},
    ]), 62, 8),
    # sizes in multiples of 16, pages of 64: heads of 64 and of 128 with values as wide (the tensor-core attention in
    # bfloat16), a window of 33 that keeps 70 (more than a page, more than the window), parts of 64 channels (the tensor-core
    # gates and the one-kernel step)
    "C": (dict(width=128, vocab=300, eps=1e-6, layers=[
        {**att(4, 2, 64, 64, 0.15, (10000.0, 32, (3.0, 200.0, 8.0, 1.0)), (33, 70), 6.0), "mlp": moe(8, 3, 32, 0.9, (64, 0.7))},
        {**rec(256, 4, 3), "mlp": moe(8, 2, 48, 0.9, (32, 0.7))},
        {**att(2, 1, 128, 128, 0.1, (300000.0, 128), (90, 5)), "mlp": moe(6, 2, 64, 1.2)},
        {**rec(96, 2, 4), "mlp": None},
        {**att(3, 3, 64, 64, 0.2, (1000.0, 64), None, 9.0), "mlp": None},
    ]), 63, 64),
    # every position sees itself and the first 25 tokens; parts of 3 channels; one layer with everything a feed-forward has
    "D": (dict(width=32, vocab=50, eps=1e-5, layers=[
        {**att(2, 1, 12, 10, 0.4, (30.0, 12, (2.0, 16.0, 2.0, 1.0)), (1, 25), 4.0), "mlp": moe(4, 2, 24, 0.5, (12, 0.8))},
        {**rec(24, 8, 2), "mlp": None},
    ]), 64, 16),
}

# how much larger than the base deviation a tensor's entries are (by the end of its name)
BOOST = {"embed": 20.0, ".gate": 3.0, ".up": 3.0, ".g": 4.0, ".y": 3.0, ".x": 3.0, ".ra": 3.0, ".ri": 3.0, "head": 3.0}


def tiny_config(name: str):
    return make_config(**TINY[name][0])


def page_size(name: str) -> int:
    return TINY[name][2]


def tiny_tensors(cfg, seed: int, std: float = 0.05) -> dict[str, torch.Tensor]:
    tensors = random_tensors(cfg, seed, std)
    g = torch.Generator().manual_seed(seed + 1000)
    rnd = lambda t, s: s * torch.randn(t.shape, generator=g)
    for n, t in tensors.items():
        if not t.dtype.is_floating_point:
            continue
        if n.endswith((".norm1", ".norm2")) or n == "final.norm":     # stored around zero: the scale is 1 + w
            new = rnd(t, 0.3)
        elif n.endswith(".norm"):                    # the norms of q and k: plain scales around one
            new = 1.0 + rnd(t, 0.3)
        elif n.endswith(".b"):                       # projection, filter and gate biases
            new = rnd(t, 0.3)
        elif n.endswith(".conv"):
            new = rnd(t, 0.5)
        elif n.endswith(".lam"):                     # memories from a few tokens to hundreds
            new = 6.0 * torch.rand(t.shape, generator=g) - 6.5
        else:
            new = t.float()
            for end, f in BOOST.items():
                if n.endswith(end):
                    new = new * f
        tensors[n] = new.to(t.dtype)
    return tensors


def make_tiny_folder(name: str, base, std: float = 0.05) -> str:
    kw, seed, _ = TINY[name]
    folder = os.path.join(str(base), f"suranex_{name}")
    if os.path.exists(os.path.join(folder, "model.safetensors")):
        return folder
    cfg = make_config(**kw)
    from turingserve_b200.config.registry import get_architecture
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w", encoding="utf-8") as f:
        json.dump(get_architecture("Suranex").to_config_json(cfg), f)
    save_file(tiny_tensors(cfg, seed, std), os.path.join(folder, "model.safetensors"))
    return folder


def random_ids(n: int, vocab: int, seed: int) -> list[int]:
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()
