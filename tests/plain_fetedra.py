"""Plain, slow Fetedra: one function per mechanism, whole sequences, no cache, nothing shared with the product.

Everything runs in the type of the tensors it is given (the tests hand it float64 or float32).  ``forward`` takes
the configuration as config.json spells it and the tensors by their checkpoint names.
"""

from __future__ import annotations

import json
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


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# -- the time mixer ------------------------------------------------------------------------------------------------------
def shifted_mix(h: torch.Tensor, mu: torch.Tensor) -> torch.Tensor:
    """Row t: h_t + (h_(t-1) - h_t) * mu, zeros before the first row."""
    before = torch.zeros_like(h)
    before[1:] = h[:-1]
    return h + (before - h) * mu


def decay_of(mix: torch.Tensor, w1: torch.Tensor, w2: torch.Tensor, w0: torch.Tensor) -> torch.Tensor:
    """exp(-exp(w2 tanh(w1 mix) + w0)), one number per channel of a row."""
    return torch.exp(-torch.exp(torch.tanh(mix @ w1.T) @ w2.T + w0))


def fading_state_scan(r, k, v, w, u, S=None):
    """r, k, w [T, H, D], v [T, H, V], u [H, D]; per head o_t = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T.
    Returns (o [T, H, V], the last states [H, D, V])."""
    T, H, D = r.shape
    V = v.shape[2]
    states = [torch.zeros(D, V, dtype=r.dtype) if S is None else S[h].clone() for h in range(H)]
    out = torch.zeros(T, H, V, dtype=r.dtype)
    for h in range(H):
        for t in range(T):
            kv = torch.outer(k[t, h], v[t, h])
            out[t, h] = (states[h] + u[h][:, None] * kv).T @ r[t, h]
            states[h] = w[t, h][:, None] * states[h] + kv
    return out, torch.stack(states)


def wkv_mixer(h: torch.Tensor, W: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    mix = {s: shifted_mix(h, W[f"{p}mu.{s}"]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ W[p + s].T).view(T, H, D) for s in "rkv")
    w = decay_of(mix["w"], W[p + "w1"], W[p + "w2"], W[p + "w0"]).view(T, H, D)
    o, _ = fading_state_scan(r, k, v, w, W[p + "u"])
    o = unit_rms(o, eps).reshape(T, H * D) * W[p + "norm"] * silu(mix["g"] @ W[p + "g"].T)
    return o @ W[p + "o"].T


# -- latent attention ------------------------------------------------------------------------------------------------------
def rotate_halves(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, ..., R]: dimension i < dims/2 turned with dimension i + dims/2 by position * base^(-2i/dims)."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    a = (positions.to(x.dtype)[:, None] * f).view([x.shape[0]] + [1] * (x.dim() - 2) + [half])
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., dims:]], -1)


def visible(T: int, window: int | None) -> torch.Tensor:
    """[T, T]: row i sees column j."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & ((d < window) if window else True)


def sink_softmax(s: torch.Tensor, ok: torch.Tensor, sink) -> torch.Tensor:
    """Weights of the keys: exp(s) over the sum of the visible ones and exp(sink)."""
    s = s.masked_fill(~ok, float("-inf"))
    top = torch.maximum(s.max(-1, keepdim=True).values, torch.as_tensor(sink, dtype=s.dtype))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def latent_attention(h: torch.Tensor, W: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, R, V, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    base, dims = float(m["rot"]["base"]), int(m["rot"]["dims"])
    q = ((unit_rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T).view(T, H, D + R)
    both = h @ W[p + "dkv"].T
    c = unit_rms(both[:, :rank], eps) * W[p + "dkv.norm"]
    k_rot = rotate_halves(both[:, rank:], pos, base, dims)
    q_rot = rotate_halves(q[..., D:], pos, base, dims)
    k = (c @ W[p + "uk"].T).view(T, H, D)
    v = (c @ W[p + "uv"].T).view(T, H, V)
    ok = visible(T, (m.get("mask") or {}).get("size"))
    gate = torch.sigmoid(h @ W[p + "g"].T)
    heads = []
    for a in range(H):
        s = (q[:, a, :D] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * float(m["scale"])
        heads.append((sink_softmax(s, ok, W[p + "sink"][a]) @ v[:, a]) * gate[:, a:a + 1])
    return torch.cat(heads, -1) @ W[p + "o"].T


# -- feed-forwards -----------------------------------------------------------------------------------------------------------
def dense_ff(h: torch.Tensor, W: dict, p: str) -> torch.Tensor:
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def clamped_expert(h: torch.Tensor, W: dict, p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ W[p + "gate"].T, max=limit)
    u = torch.clamp(h @ W[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def choose(scores: torch.Tensor, correction: torch.Tensor, top: int, groups: int, keep: int):
    """One token's experts, best first: the ``top`` largest scores + correction among the ``keep`` groups of neighbours
    whose two largest such numbers have the largest sum."""
    by = (scores + correction).tolist()
    size = len(by) // groups
    strength = [sum(sorted(by[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: -strength[g])[:keep]
    open_ = [e for e in range(len(by)) if e // size in kept]
    return sorted(open_, key=lambda e: -by[e])[:top]


def routed_ff(h: torch.Tensor, W: dict, p: str, f: dict) -> torch.Tensor:
    router = f["router"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    s = torch.sigmoid(h @ W[p + "router"].T)
    out = torch.zeros(h.shape[0], W[p + "e0.down"].shape[0], dtype=h.dtype)
    for t in range(h.shape[0]):
        idx = choose(s[t], W[p + "correction"], int(router["top"]), int(groups["count"]), int(groups["keep"]))
        total = sum(s[t, e] for e in idx) + 1e-20
        for e in idx:
            weight = s[t, e] / total * float(router["scale"])
            out[t] += weight * clamped_expert(h[t:t + 1], W, f"{p}e{e}.", float(f["expert"]["limit"]))[0]
    if f.get("shared"):
        share = torch.sigmoid(h @ W[p + "shared.sg"].T)
        out = out + share * clamped_expert(h, W, p + "shared.", float(f["shared"]["limit"]))
    return out


# -- the stream in copies ----------------------------------------------------------------------------------------------------
def read_streams(xs: list, w_in: torch.Tensor) -> torch.Tensor:
    return sum(w_in[s] * xs[s] for s in range(len(xs)))


def write_streams(xs: list, y: torch.Tensor, w_mix: torch.Tensor, w_out: torch.Tensor) -> list:
    """The new copies, all from the old ones; the mix is indexed [from, to]."""
    n = len(xs)
    return [sum(w_mix[s, t] * xs[s] for s in range(n)) + w_out[t] * y for t in range(n)]


# -- the model ---------------------------------------------------------------------------------------------------------------
MIXERS = {"wkv": wkv_mixer, "latent_attention": latent_attention}


def forward(config: dict, W: dict, tokens, after: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one whole sequence; ``after`` receives the sum of the streams after every layer."""
    eps = float(config["norm"]["eps"])
    x0 = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    S = config.get("streams")
    xs = [x0.clone() for _ in range(S or 1)]
    for i, entry in enumerate(config["layers"]):
        pre = f"l{i}."
        subs = [(1, lambda u: MIXERS[entry["type"]](u, W, pre + "mix.", entry["mixer"], eps))]
        if entry.get("mlp"):
            f = entry["mlp"]
            subs.append((2, lambda u: dense_ff(u, W, pre + "mlp.") if f["kind"] == "dense" else routed_ff(u, W, pre + "mlp.", f)))
        for q, fn in subs:
            w = W[f"{pre}norm{q}"]
            if S:
                hc = f"{pre}hc{q}."
                y = fn(zero_centred_norm(read_streams(xs, W[hc + "in"]), w, eps))
                xs = write_streams(xs, y, W[hc + "mix"], W[hc + "out"])
            else:
                xs = [xs[0] + fn(zero_centred_norm(xs[0], w, eps))]
        if after is not None:
            after.append(sum(xs))
    return (zero_centred_norm(sum(xs), W["final.norm"], eps) @ W["embed"].T) * float(config.get("logit_scale", 1.0))
