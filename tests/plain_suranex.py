"""Plain, slow Suranex: one function per mechanism, whole sequences, no cache, nothing shared with the product.

Everything runs in the type of the tensors it is given (the tests hand it float64 or float32).  ``forward`` takes
the configuration as config.json spells it and the tensors by their checkpoint names.
"""

from __future__ import annotations

import json
import math
import os

import torch
from safetensors.torch import load_file


def read_folder(folder: str, dtype=torch.float64):
    with open(os.path.join(folder, "config.json"), encoding="utf-8") as f:
        cfg = json.load(f)
    tensors = load_file(os.path.join(folder, "model.safetensors"))
    return cfg, {k: (v.to(dtype) if v.dtype.is_floating_point else v) for k, v in tensors.items()}


# -- norms and activations -------------------------------------------------------------------------------------------
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last dimension, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm whose stored weight lies around zero: the scale is 1 + w."""
    return unit_rms(x, eps) * (1.0 + w)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


# -- rotation ----------------------------------------------------------------------------------------------------------
def plain_frequencies(base: float, dims: int) -> list[float]:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def key_frequencies(base: float, dims: int, scaling: dict | None) -> tuple[list[float], float]:
    """(frequencies, magnitude of cosine and sine).  With ``scaling`` the plain frequency of a pair that turns often
    within ``original`` positions stays, one that turns rarely is slowed by ``factor``, a linear ramp between."""
    f = plain_frequencies(base, dims)
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def where(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first = max(math.floor(where(float(scaling["fast"]))), 0)
    last = min(math.ceil(where(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, freqs: list[float], magnitude: float = 1.0,
                  sign: float = 1.0) -> torch.Tensor:
    """x [T, heads, D]: dimension i turned with dimension i + n, n = len(freqs), by sign * position * f_i; the
    dimensions from 2 n on pass."""
    out = x.clone()
    n = len(freqs)
    ang = positions.to(x.dtype)[:, None] * torch.tensor(freqs, dtype=x.dtype)[None, :] * sign
    c, s = torch.cos(ang)[:, None, :] * magnitude, torch.sin(ang)[:, None, :] * magnitude
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


# -- attention ---------------------------------------------------------------------------------------------------------
def visible(T: int, mask: dict | None) -> torch.Tensor:
    """[T, T] booleans: the query (row) sees the key (column): never a later one; with a window of ``size`` the last
    ``size`` positions up to its own, and the first ``keep_first`` of the sequence whatever the distance."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    if mask:
        ok = ok & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0))))
    return ok


def softmax_attention(q, k, v, scale: float, softcap, mask) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]."""
    T, H, _ = q.shape
    G = k.shape[1]
    ok = visible(T, mask)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        out[:, h] = torch.softmax(s.masked_fill(~ok, float("-inf")), -1) @ v[:, g]
    return out


def attention_mixer(h: torch.Tensor, W: dict, p: str, m: dict, eps: float, positions: torch.Tensor) -> torch.Tensor:
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    V = m.get("vdim", D)
    q = unit_rms((h @ W[p + "q"].T).view(T, H, D), eps) * W[p + "q.norm"]
    k = unit_rms((h @ W[p + "k"].T).view(T, G, D), eps) * W[p + "k.norm"]
    v = unit_rms((h @ W[p + "v"].T).view(T, G, V), eps)
    rot = m.get("rot")
    if rot:
        base = float(rot["base"])
        f, mag = key_frequencies(base, int(rot["dims"]), rot.get("scaling"))
        q, k = rotate_halves(q, positions, f, mag), rotate_halves(k, positions, f, mag)
        fv = plain_frequencies(base, V)
        v = rotate_halves(v, positions, fv)
    a = softmax_attention(q, k, v, float(m["scale"]), m.get("softcap"), m.get("mask"))
    if rot:
        a = rotate_halves(a, positions, fv, sign=-1.0)
    a = a * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return a.reshape(T, H * V) @ W[p + "o"].T


# -- the real-gated linear recurrent unit --------------------------------------------------------------------------------
def causal_filter(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """x [T, C], w [C, taps] (the last column is the present token's), zeros before the start."""
    T, C = x.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x])
    out = b.expand(T, C).clone()
    for j in range(taps):
        out = out + padded[j:j + T] * w[:, j]
    return out


def block_gate(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """sigmoid of a block-diagonal product: u [T, C] in w.shape[0] equal parts, part n through w[n] [out, in]."""
    n, size, _ = w.shape
    parts = [u[:, i * size:(i + 1) * size] @ w[i].T + b[i] for i in range(n)]
    return torch.sigmoid(torch.cat(parts, dim=1))


def gated_recurrence(u, r, i, lam) -> torch.Tensor:
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a = -8 r softplus(lam), from S = 0."""
    log_a = -8.0 * r * softplus(lam)
    a = torch.exp(log_a)
    add = torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    S = torch.zeros_like(u[0])
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + add[t]
        out[t] = S
    return out


def rglru_mixer(h: torch.Tensor, W: dict, p: str, m: dict) -> torch.Tensor:
    y = gelu_tanh(h @ W[p + "y"].T + W[p + "y.b"])
    u = causal_filter(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    r = block_gate(u, W[p + "ra"], W[p + "ra.b"])
    i = block_gate(u, W[p + "ri"], W[p + "ri.b"])
    return (gated_recurrence(u, r, i, W[p + "lam"]) * y) @ W[p + "o"].T


# -- feed-forward --------------------------------------------------------------------------------------------------------
def clamped_expert(x: torch.Tensor, W: dict, p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(x @ W[p + "gate"].T, max=limit)
    u = torch.clamp(x @ W[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def table_moe(x: torch.Tensor, ids: torch.Tensor, W: dict, p: str, f: dict) -> torch.Tensor:
    """Every token's experts are its id's row of a table, with equal weights; a shared expert is added."""
    chosen = W[p + "table"].long()[ids]                                     # [T, top]
    out = torch.zeros_like(x)
    for e in range(int(f["router"]["experts"])):
        rows = (chosen == e).any(dim=1)
        if rows.any():
            out[rows] += clamped_expert(x[rows], W, f"{p}e{e}.", float(f["expert"].get("limit", math.inf))) / chosen.shape[1]
    if f.get("shared"):
        out = out + clamped_expert(x, W, p + "shared.", float(f["shared"].get("limit", math.inf)))
    return out


# -- the model -----------------------------------------------------------------------------------------------------------
def forward(cfg: dict, W: dict, ids, layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab].  ``layers_out`` receives the stream after every layer."""
    ids = torch.as_tensor(ids, dtype=torch.long)
    positions = torch.arange(len(ids))
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][ids]
    for n, entry in enumerate(cfg["layers"]):
        p = f"l{n}."
        if entry["type"] == "attention":
            y = attention_mixer(x, W, p + "mix.", entry["mixer"], eps, positions)
        else:
            y = rglru_mixer(x, W, p + "mix.", entry["mixer"])
        x = x + zero_centred_norm(y, W[p + "norm1"], eps)
        if entry.get("mlp"):
            x = x + zero_centred_norm(table_moe(x, ids, W, p + "mlp.", entry["mlp"]), W[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return zero_centred_norm(x, W["final.norm"], eps) @ W["head"].T


def greedy(cfg: dict, W: dict, prompt: list[int], n: int) -> list[int]:
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(forward(cfg, W, ids)[-1].argmax()))
    return ids[len(prompt):]
