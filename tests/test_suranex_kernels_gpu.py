"""The kernels Suranex brings, each alone against the plain functions: norms of outputs from every form of output, normed
and turned heads with their cache write, attention behind a window that keeps the first tokens with outputs turned back
and gated, the real-gated recurrent unit (filter, gates, scan, the one-kernel step), experts chosen by a table and the
clamped gated unit."""

from __future__ import annotations

import math
from types import SimpleNamespace

import pytest
import torch

from tests import plain_suranex as plain

pytestmark = pytest.mark.gpu
DEV = "cuda"


@pytest.fixture(scope="module")
def ops():
    from turingserve_b200 import kernels
    kernels.use(None)
    return kernels.ops()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def tol(dtype):
    return dict(rtol=2e-2, atol=2e-2) if dtype == torch.bfloat16 else dict(rtol=2e-5, atol=2e-5)


def close(got, want, dtype, slack=1.0):
    lim = {k: v * slack for k, v in tol(dtype).items()}
    return torch.allclose(got.double().cpu(), want.double().cpu(), **lim)


DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


# -- the norm of what a sublayer returns -------------------------------------------------------------------------------
def plain_update(stream, y, w, eps):
    return stream.double() + plain.unit_rms(y.double(), eps) * w.double()


@DTYPES
@pytest.mark.parametrize("T,h", [(1, 40), (3, 72), (5, 1536), (70, 2500), (2, 3584), (3, 4100), (4, 33)])
def test_output_norm_of_a_tensor(ops, dtype, T, h):
    """Added to the stream, started from the embedding rows, and with the norm that reads the stream next; row lengths the
    register kernel takes and others."""
    g = torch.Generator(device=DEV).manual_seed(h)
    y = (torch.randn(T, h, generator=g, device=DEV) * 5).to(dtype)
    w, w2 = torch.randn(h, generator=g, device=DEV) + 1, torch.randn(h, generator=g, device=DEV) + 1
    old = torch.randn(T, h, generator=g, device=DEV) * 3
    base = torch.randn(T, h, generator=g, device=DEV).to(dtype)
    for b in (None, base):
        for nw in (None, w2):
            stream, out = old.clone(), torch.empty(T, h, dtype=dtype, device=DEV)
            ops.post_norm(out, stream, y, w, 0.3, base=b, next_weight=nw, next_eps=0.7)
            want = plain_update(old if b is None else b, y, w, 0.3)
            assert torch.allclose(stream.double(), want, rtol=1e-5, atol=1e-5)          # (32-bit in both engine types)
            read = want if nw is None else plain.unit_rms(want, 0.7) * w2.double()
            assert close(out, read, dtype)


def test_output_norm_takes_eps_inside_the_root(ops):
    y = torch.full((1, 8), 1.0, device=DEV)
    stream, out = torch.zeros(1, 8, device=DEV), torch.empty(1, 8, device=DEV)
    ops.post_norm(out, stream, y, torch.full((8,), 2.0, device=DEV), 3.0)
    assert torch.allclose(out, torch.ones_like(out)) and torch.equal(out, stream)       # 1 / sqrt(1 + 3) * 2


@pytest.mark.parametrize("T", [1, 8, 40])
@pytest.mark.parametrize("h", [1536, 200])
def test_output_norm_of_a_product_left_unreduced(ops, T, h):
    from turingserve_b200 import kernels
    g = torch.Generator(device=DEV).manual_seed(T)
    K = 1024
    x = torch.randn(T, K, generator=g, device=DEV).to(torch.bfloat16)
    wt = (torch.randn(h, K, generator=g, device=DEV) * 0.1).to(torch.bfloat16)
    bias = torch.randn(h, generator=g, device=DEV).to(torch.bfloat16)
    w = torch.ones(h, device=DEV)
    for b in (None, bias):
        y = ops.linear(torch.empty(T, h, dtype=torch.bfloat16, device=DEV), x, wt, b, may_defer=True)
        assert isinstance(y, (kernels.LazyProduct, kernels.Deferred))
        stream, out = torch.zeros(T, h, device=DEV), torch.empty(T, h, dtype=torch.bfloat16, device=DEV)
        ops.post_norm(out, stream, y, w, 1e-6)
        full = x.double() @ wt.double().T + (0.0 if b is None else b.double())
        assert torch.allclose(stream.double(), plain_update(torch.zeros_like(full), full, w, 1e-6), rtol=1e-4, atol=1e-4)


@DTYPES
@pytest.mark.parametrize("T,h,top", [(3, 72, 2), (9, 1536, 3), (2, 33, 1), (5, 4100, 4)])
def test_output_norm_of_a_routed_sum(ops, dtype, T, h, top):
    """scale times the sum of a token's rows at their sorted places, with and without weights, with and without the output
    of an expert that every token uses."""
    g = torch.Generator(device=DEV).manual_seed(h + top)
    rows = torch.randn(T * top, h, generator=g, device=DEV)
    place = torch.randperm(T * top, generator=torch.Generator().manual_seed(1)).to(torch.int32).to(DEV)
    weights = torch.rand(T, top, generator=g, device=DEV)
    add = torch.randn(T, h, generator=g, device=DEV).to(dtype)
    w, old = torch.randn(h, generator=g, device=DEV), torch.randn(T, h, generator=g, device=DEV)
    for pw in (None, weights):
        for extra in (None, add):
            chosen = rows[place.long()].view(T, top, h).double()
            y = 0.25 * (chosen if pw is None else chosen * pw.double()[..., None]).sum(1)
            if extra is not None:
                y = y + extra.double()
            stream, out = old.clone(), torch.empty(T, h, dtype=dtype, device=DEV)
            ops.post_norm(out, stream, extra, w, 1e-5, rows=rows, place=place, pair_weights=pw, top=top, scale=0.25)
            want = plain_update(old, y, w, 1e-5)
            assert torch.allclose(stream.double(), want, rtol=1e-5, atol=1e-5) and close(out, want, dtype)


# -- normed and turned heads, cache write ------------------------------------------------------------------------------
def freq_tensor(f):
    return torch.tensor(f, dtype=torch.float64).float().to(DEV)


@DTYPES
@pytest.mark.parametrize("H,G,D,V,rot,page,norms,v_norm,turned", [
    (4, 2, 16, 8, 8, 16, True, True, True), (3, 3, 24, 40, 24, 8, True, True, True), (7, 1, 128, 72, 48, 64, True, True, True),
    (2, 1, 12, 20, 0, 4, True, False, False), (5, 5, 10, 6, 6, 16, False, True, True), (8, 2, 64, 64, 64, 32, True, True, True),
    (2, 1, 256, 64, 128, 16, True, True, False), (3, 1, 192, 256, 64, 8, False, False, True), (6, 2, 128, 128, 128, 16, True, True, True),
    (1, 1, 200, 30, 100, 16, True, True, True), (9, 3, 32, 16, 0, 16, True, True, True)])
def test_heads_are_normed_turned_and_cached(ops, dtype, H, G, D, V, rot, page, norms, v_norm, turned):
    g = torch.Generator(device=DEV).manual_seed(H * D + V)
    T, eps, mag = 19, 1e-3, 1.25
    positions = [0, 1, 2, 63, 64, 65, 999, 4095, 4096] + list(range(300, 310))
    k_off, v_off = H * D, (H + G) * D
    width = v_off + G * V + H
    proj = (torch.randn(T, -(-width // 8) * 8 + 8, generator=g, device=DEV) * 3).to(dtype)[:, :width]
    before = proj.clone()
    q_w, k_w = ((torch.randn(D, generator=g, device=DEV) + 1) if norms else None for _ in range(2))
    fk, fv = plain.plain_frequencies(500.0, rot) if rot else [], plain.plain_frequencies(90.0, V) if turned else []
    pages = 7
    k_cache = torch.full((pages, G, page, D), 9.0, dtype=dtype, device=DEV)
    v_cache = torch.full((pages, G, page, V), 9.0, dtype=dtype, device=DEV)
    slots = torch.randperm(pages * page, generator=torch.Generator().manual_seed(3))[:T].to(torch.int32)
    slots[5] = -1                                                     # a row that caches nothing
    ops.qkv_heads_write(proj, k_off, v_off, i32(positions), q_w, k_w, eps, freq_tensor(fk) if rot else None, mag, rot, v_norm,
                        freq_tensor(fv) if turned else None, k_cache, v_cache, slots.to(DEV), H, G, D, V, page)
    b, pos = before.double().cpu(), torch.tensor(positions)
    parts = {"q": b[:, :k_off].view(T, H, D), "k": b[:, k_off:v_off].view(T, G, D), "v": b[:, v_off:v_off + G * V].view(T, G, V)}
    for name, w in (("q", q_w), ("k", k_w)):
        if norms:
            parts[name] = plain.unit_rms(parts[name], eps) * w.double().cpu()
        if rot:
            parts[name] = plain.rotate_halves(parts[name], pos, fk, mag)
    if v_norm:
        parts["v"] = plain.unit_rms(parts["v"], eps)
    if turned:
        parts["v"] = plain.rotate_halves(parts["v"], pos, fv)
    for t in range(T):
        slack = 1.0 + positions[t] / 20.0 if dtype == torch.float32 else 1.0 + positions[t] / 1000.0
        big = 3.0 if not norms else 1.0
        assert close(proj[t, :k_off].view(H, D), parts["q"][t], dtype, slack * big), t
        s = int(slots[t])
        if s >= 0:
            assert close(k_cache[s // page, :, s % page], parts["k"][t], dtype, slack * big), t
            assert close(v_cache[s // page, :, s % page], parts["v"][t], dtype, slack * (1.0 if v_norm else 3.0)), t
    assert torch.equal(proj[:, k_off:], before[:, k_off:])            # keys, values and gates of the input stay
    written = torch.zeros(pages * page, dtype=torch.bool)
    written[slots[slots >= 0].long()] = True
    for cache, n in ((k_cache, D), (v_cache, V)):
        rest = cache.permute(0, 2, 1, 3).reshape(pages * page, G * n)[~written.to(DEV)]
        assert float((rest.float() - 9.0).abs().max()) == 0.0
    again = before.clone()
    ops.qkv_heads_write(again, k_off, v_off, i32(positions), q_w, k_w, eps, freq_tensor(fk) if rot else None, mag, rot, v_norm,
                        freq_tensor(fv) if turned else None, None, None, None, H, G, D, V, page)
    assert torch.equal(again[:, :k_off], proj[:, :k_off])             # without slots q is the same


@pytest.mark.parametrize("T", [1, 8, 33, 100])
@pytest.mark.parametrize("H,G,D,V,rot", [(6, 2, 128, 64, 32), (12, 2, 128, 128, 128), (5, 5, 64, 64, 64), (3, 3, 24, 48, 16)])
def test_a_projection_left_unreduced_is_finished_by_the_heads_kernel(ops, T, H, G, D, V, rot):
    """The same bits in q, in both caches and in the gate columns behind the values as the finished product gives."""
    from turingserve_b200 import kernels
    g = torch.Generator(device=DEV).manual_seed(T + D)
    K, page = 1536, 16
    v_off = (H + G) * D
    N = -(-(v_off + G * V + H) // 8) * 8
    x = torch.randn(T, K, generator=g, device=DEV).to(torch.bfloat16)
    w = (torch.randn(N, K, generator=g, device=DEV) * 0.05).to(torch.bfloat16)
    hw = torch.randn(D, generator=g, device=DEV)
    fk, fv = freq_tensor(plain.plain_frequencies(1000.0, rot)), freq_tensor(plain.plain_frequencies(1000.0, V))
    pos, slots = i32([700 + 3 * t for t in range(T)]), i32([page + 2 * t for t in range(T)])
    results = []
    for defer in (False, True):
        out = torch.zeros(T, N, dtype=torch.bfloat16, device=DEV)
        kc = torch.zeros(3 + 2 * T // page, G, page, D, dtype=torch.bfloat16, device=DEV)
        vc = torch.zeros(3 + 2 * T // page, G, page, V, dtype=torch.bfloat16, device=DEV)
        proj = ops.linear(out, x, w, may_defer=defer, lazy=False)
        assert isinstance(proj, kernels.Deferred) == defer
        proj = ops.qkv_heads_write(proj, H * D, v_off, pos, hw, hw, 1e-6, fk, 1.1, rot, True, fv, kc, vc, slots, H, G, D, V, page)
        results.append((proj[:, :H * D].clone(), proj[:, v_off + G * V:].clone(), kc, vc))
    for a, b in zip(*results):
        assert torch.equal(a, b)
    assert float(results[0][2].abs().max()) > 0 and float(results[0][3].abs().max()) > 0


# -- attention: window with kept first tokens, cap, outputs turned back and gated -------------------------------------------
def paged(rows, page, order):
    T, G, D = rows.shape
    cache = torch.zeros(max(order) + 1, G, page, D, dtype=rows.dtype, device=DEV)
    for p, at in enumerate(order):
        part = rows[p * page:(p + 1) * page]
        cache[at, :, :part.shape[0]] = part.transpose(0, 1)
    return cache


def batch(q_lens, seq_lens):
    starts = [0]
    for n in q_lens:
        starts.append(starts[-1] + n)
    return SimpleNamespace(q_start=i32(starts), seq_lens=i32(seq_lens), num_requests=len(q_lens),
                           num_decode=sum(1 for n in q_lens if n == 1), max_q_len=max(q_lens), max_seq_len=max(seq_lens))


def run_attention(ops, q, ks, vs, q_lens, page, scale, cap, window, keep, v_freqs, gate):
    """q [T, H, D] for all requests; ks, vs: every request's rows up to its length; pages in a shuffled pool."""
    G, V = ks[0].shape[1], vs[0].shape[2]
    rng = torch.Generator().manual_seed(len(ks))
    n_pages = [-(-k.shape[0] // page) for k in ks]
    order = (torch.randperm(sum(n_pages), generator=rng) + 1).tolist()
    kc = torch.zeros(sum(n_pages) + 1, G, page, q.shape[2], dtype=q.dtype, device=DEV)
    vc = torch.zeros(sum(n_pages) + 1, G, page, V, dtype=q.dtype, device=DEV)
    bt = torch.zeros(len(ks), max(n_pages), dtype=torch.int32)
    at = 0
    for r, (k, v, n) in enumerate(zip(ks, vs, n_pages)):
        mine = order[at:at + n]
        at += n
        bt[r, :n] = torch.tensor(mine)
        for pool, rows in ((kc, k), (vc, v)):
            one = paged(rows, page, mine)
            for p in mine:
                pool[p] = one[p]
    out = torch.empty(q.shape[0], q.shape[1], V, dtype=q.dtype, device=DEV)
    ops.attention_biased(out, q, kc, vc, bt.to(DEV), batch(q_lens, [k.shape[0] for k in ks]), G, page, scale, cap, None, window,
                         keep=keep, out_freq=freq_tensor(v_freqs) if v_freqs else None, gate=gate)
    return out


def plain_attention(q, k, v, scale, cap, window, keep, v_freqs, gate):
    """The last q.shape[0] positions of a sequence, in 64-bit."""
    T, n = k.shape[0], q.shape[0]
    H, G = q.shape[1], k.shape[1]
    mask = {"size": window, "keep_first": keep} if window else None
    ok = plain.visible(T, mask)[T - n:]
    kk, vv = (x.double().cpu().repeat_interleave(H // G, dim=1) for x in (k, v))
    s = torch.einsum("ihd,jhd->hij", q.double().cpu(), kk) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    o = torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~ok[None], -math.inf), -1), vv)
    if v_freqs:
        o = plain.rotate_halves(o, torch.arange(T - n, T), v_freqs, sign=-1.0)
    return o if gate is None else o * torch.sigmoid(gate.double().cpu())[:, :, None]


KINDS = pytest.mark.parametrize("dtype,H,G,D,V,page", [
    (torch.float32, 4, 2, 16, 8, 16), (torch.float32, 3, 1, 12, 40, 8), (torch.float32, 5, 5, 64, 64, 64),
    (torch.bfloat16, 6, 2, 64, 64, 16), (torch.bfloat16, 3, 1, 128, 128, 64), (torch.bfloat16, 4, 2, 40, 24, 8),
    (torch.bfloat16, 24, 1, 64, 64, 32), (torch.bfloat16, 40, 1, 128, 128, 16)])


@KINDS
@pytest.mark.parametrize("window,keep", [(None, 0), (1, 0), (1, 9), (30, 5), (64, 64), (100, 70), (33, 200), (70, 0)])
@pytest.mark.parametrize("splits", [0, 1, 3])
def test_attention_in_batches_of_unequal_requests(ops, dtype, H, G, D, V, page, window, keep, splits):
    """Single tokens and portions of unequal requests in one launch, windows that end inside, at and past tiles, kept
    tokens that reach into the window, lie far before it and cover more than a tile; gates in columns of a wider tensor."""
    g = torch.Generator(device=DEV).manual_seed(H * D + (window or 0))
    q_lens, seq_lens = [1, 1, 1, 1, 2, 90, 7], [1, 64, 333, 129, 71, 300, 7]
    T = sum(q_lens)
    q = (torch.randn(T, H, D, generator=g, device=DEV)).to(dtype)
    ks = [torch.randn(n, G, D, generator=g, device=DEV).to(dtype) for n in seq_lens]
    vs = [torch.randn(n, G, V, generator=g, device=DEV).to(dtype) for n in seq_lens]
    gate = torch.randn(T, H + 16, generator=g, device=DEV).to(dtype)[:, 8:8 + H]
    fv = plain.plain_frequencies(40.0, V)
    scale, cap = 1.5 / math.sqrt(D), 2.5
    old = ops.biased_decode_splits
    ops.biased_decode_splits = splits
    try:
        got = run_attention(ops, q, ks, vs, q_lens, page, scale, cap, window, keep, fv, gate)
        bare = run_attention(ops, q, ks, vs, q_lens, page, scale, 0.0, window, keep, None, None)
    finally:
        ops.biased_decode_splits = old
    at = 0
    for r, n in enumerate(q_lens):
        rows = slice(at, at + n)
        at += n
        want = plain_attention(q[rows], ks[r], vs[r], scale, cap, window, keep, fv, gate[rows])
        assert close(got[rows], want, dtype, 2.0), (r, float((got[rows].double().cpu() - want).abs().max()))
        assert close(bare[rows], plain_attention(q[rows], ks[r], vs[r], scale, 0.0, window, keep, None, None), dtype, 2.0), r


@pytest.mark.parametrize("decode", [False, True])
@KINDS
def test_one_loud_key_at_every_edge(ops, decode, dtype, H, G, D, V, page):
    """Every key is silent but one, whose value is marked: the query finds it exactly where the window and the kept first
    tokens let it, just inside and just outside both, at page borders, and never one place ahead of itself."""
    marked = 3
    for T, window, keep in ((700, 100, 37), (150, 64, 64), (321, 1, 130), (90, 200, 5), (260, 65, 0)):
        n_q = 1 if decode else 40
        i = T - 1
        places = {i, i - 1, i - window + 1, i - window, i - window - 1, keep - 1, keep, keep + 1, 0, page - 1, page,
                  (i // page) * page, (i // page) * page - 1, keep // page * page, i // 2}
        for j in sorted(p for p in places if 0 <= p <= i):
            k = torch.zeros(T, G, D, dtype=dtype, device=DEV)
            v = torch.zeros(T, G, V, dtype=dtype, device=DEV)
            k[j, :, 1] = 60.0
            v[j, :, marked] = 1.0
            q = torch.zeros(n_q, H, D, dtype=dtype, device=DEV)
            q[:, :, 1] = 1.0
            out = run_attention(ops, q, [k], [v], [n_q], page, 1.0, 0.0, window, keep, None, None)
            for row in range(n_q):
                p = T - n_q + row
                seen = j <= p and (p - j < window or j < keep)
                assert abs(float(out[row, 0, marked]) - (1.0 if seen else 0.0)) < 1e-5, (T, window, keep, j, p)


@KINDS
def test_turned_values_hold_distances_only(ops, dtype, H, G, D, V, page):
    """The same sequence of values cached at positions 0.. and at positions shifted by 500 (equal keys): what a head
    returns for a query the same distance away is the same, although every cached row differs."""
    g = torch.Generator(device=DEV).manual_seed(2)
    raw = torch.randn(30, G, V, generator=g, device=DEV)
    fv = plain.plain_frequencies(60.0, V)
    outs = []
    for shift in (0, 500):
        n = 30 + shift
        v = torch.zeros(n, G, V, device=DEV)
        v[shift:] = plain.rotate_halves(raw.double().cpu(), torch.arange(shift, n), fv).float().to(DEV)
        k, q = torch.ones(n, G, D, dtype=dtype, device=DEV), torch.ones(1, H, D, dtype=dtype, device=DEV)
        outs.append(run_attention(ops, q, [k], [v.to(dtype)], [1], page, 0.1, 0.0, 30, 0, fv, None))
    assert close(outs[0], outs[1], dtype, 10.0 if dtype == torch.float32 else 1.0)
    assert float(outs[0].float().abs().max()) > 0.1


# -- the real-gated linear recurrent unit --------------------------------------------------------------------------------
def unit_consts(g, W, blocks, taps, dtype):
    rnd = lambda *s: torch.randn(*s, generator=g, device=DEV)
    size = W // blocks
    return SimpleNamespace(
        conv=rnd(W, taps) * 0.5, conv_b=rnd(W) * 0.2, ra=(rnd(blocks, size, size) * 1.5 / math.sqrt(size)).to(dtype),
        ri=(rnd(blocks, size, size) * 1.5 / math.sqrt(size)).to(dtype), ra_b=rnd(W) * 0.5, ri_b=rnd(W) * 0.5,
        lam=6.0 * torch.rand(W, generator=g, device=DEV) - 6.5)


def plain_unit(proj, c, W, round_u=None):
    """One request's rows [T, y | x] -> (S gelu(y), final S) in 64-bit; ``round_u``: the filter's output rounded so."""
    p = proj.double().cpu()
    d = {n: getattr(c, n).double().cpu() for n in vars(c)}
    blocks, size = d["ra"].shape[:2]
    u = plain.causal_filter(p[:, W:], d["conv"], d["conv_b"])
    if round_u is not None:
        u = u.to(round_u).double()
    r = plain.block_gate(u, d["ra"], d["ra_b"].view(blocks, size))
    i = plain.block_gate(u, d["ri"], d["ri_b"].view(blocks, size))
    S = plain.gated_recurrence(u, r, i, d["lam"])
    return S * plain.gelu_tanh(p[:, :W]), S[-1]


def run_unit(ops, proj, state, c, cuts, slots, W, blocks, taps, one_kernel=True):
    """The rows of ``proj`` belong to len(slots) requests of equal length; ``cuts`` are the step sizes."""
    rate = (8.0 * torch.nn.functional.softplus(c.lam.double())).float()
    n_req, T = len(slots), proj.shape[0] // len(slots)
    out = torch.empty(proj.shape[0], W, dtype=proj.dtype, device=DEV)
    at, fused = 0, 0
    for n in cuts:
        rows = torch.cat([torch.arange(r * T + at, r * T + at + n) for r in range(n_req)]).to(DEV)
        step = SimpleNamespace(q_start=i32([i * n for i in range(n_req + 1)]), state_slots=i32(slots), num_requests=n_req,
                               token_request=i32([r for r in range(n_req) for _ in range(n)]), max_q_len=n,
                               positions=i32([at + i for _ in range(n_req) for i in range(n)]))
        p = proj[rows].contiguous()
        o = torch.empty(len(rows), W, dtype=proj.dtype, device=DEV)
        if one_kernel and ops.rglru_step(o, p, 0, W, c.conv, c.conv_b, c.ra, c.ri, c.ra_b, c.ri_b, rate, state, step, taps):
            fused += 1
        else:
            u = torch.empty(len(rows), W, dtype=proj.dtype, device=DEV)
            ops.short_filter(u, p, W, c.conv, c.conv_b, state, W, step, taps)
            ab = torch.empty(len(rows), W, 2, device=DEV)
            ops.rglru_gates(ab, u, c.ra, c.ri, c.ra_b, c.ri_b, rate)
            ops.rglru_scan(o, ab, p, 0, W, state, step, taps)
        out[rows] = o
        at += n
    assert at == T
    return out, fused


@DTYPES
@pytest.mark.parametrize("W,blocks,taps", [(60, 3, 4), (36, 1, 1), (24, 8, 2), (64, 1, 3), (256, 4, 4), (96, 2, 8), (512, 2, 2),
                                           (35, 5, 3), (640, 1, 4)])
def test_recurrent_unit_whole_in_portions_and_token_by_token(ops, dtype, W, blocks, taps):
    """The same tokens as one portion, in portions down to two tokens and one (shorter than the filter's memory), and one
    by one (through the one-kernel step where it takes the shape, and through the chain): the plain outputs, states and
    ring of inputs; requests whose slots are not their batch rows; slots of others untouched."""
    g = torch.Generator(device=DEV).manual_seed(W + taps)
    T, slots = 45, [4, 1, 6]
    c = unit_consts(g, W, blocks, taps, dtype)
    proj = torch.randn(3 * T, 2 * W, generator=g, device=DEV).to(dtype)
    wants = [plain_unit(proj[r * T:(r + 1) * T], c, W, dtype if dtype == torch.bfloat16 else None) for r in range(3)]
    width = (1 + (taps if taps > 1 else 0)) * W
    lim = dict(rtol=1e-2, atol=6e-3) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=2e-5)
    for cuts, one_kernel in (([T], True), ([16, 2, 1, 1, 5, 2, 2, 3, 13], True), ([1] * T, True), ([1] * T, False)):
        state = torch.zeros(8, width, device=DEV)
        state[0] = 7.0
        out, fused = run_unit(ops, proj, state, c, cuts, slots, W, blocks, taps, one_kernel)
        takes = dtype == torch.bfloat16 and (W // blocks) % 8 == 0
        assert fused == (sum(1 for n in cuts if n == 1) if takes and one_kernel else 0)
        for r, slot in enumerate(slots):
            mine = proj[r * T:(r + 1) * T]
            assert torch.allclose(out[r * T:(r + 1) * T].double().cpu(), wants[r][0], **lim), (cuts[:3], r)
            assert torch.allclose(state[slot, :W].double().cpu(), wants[r][1], **lim), (cuts[:3], r)
            if taps > 1:
                ring = state[slot, W:].view(taps, W)
                for t in range(T - taps + 1, T):
                    assert torch.equal(ring[t % taps], mine[t, W:].float()), (cuts[:3], t)
        assert float((state[0] - 7.0).abs().max()) == 0.0 and float(state[[2, 3, 5, 7]].abs().max()) == 0.0


@DTYPES
def test_recurrent_unit_long_portions_unequal_requests_and_many_rows(ops, dtype):
    """Requests of 1 to 700 tokens in one launch (the scan's groups of 256 tokens, its eight-token segments, single tokens
    beside portions), each against itself alone in other cuts; eleven single tokens (more than a block takes)."""
    g = torch.Generator(device=DEV).manual_seed(4)
    W, blocks, taps = 128, 2, 3
    c = unit_consts(g, W, blocks, taps, dtype)
    lens = [1, 700, 9, 256, 257, 8, 1, 30]
    proj = torch.randn(sum(lens), 2 * W, generator=g, device=DEV).to(dtype)
    rate = (8.0 * torch.nn.functional.softplus(c.lam.double())).float()
    starts = [sum(lens[:i]) for i in range(len(lens) + 1)]
    state = torch.zeros(9, 4 * W, device=DEV)
    slots = [3, 0, 7, 1, 5, 2, 8, 4]
    step = SimpleNamespace(q_start=i32(starts), state_slots=i32(slots), num_requests=len(lens), max_q_len=max(lens),
                           token_request=i32([r for r, n in enumerate(lens) for _ in range(n)]),
                           positions=i32([i for n in lens for i in range(n)]))
    u, o = (torch.empty(sum(lens), W, dtype=dtype, device=DEV) for _ in range(2))
    ab = torch.empty(sum(lens), W, 2, device=DEV)
    ops.short_filter(u, proj, W, c.conv, c.conv_b, state, W, step, taps)
    ops.rglru_gates(ab, u, c.ra, c.ri, c.ra_b, c.ri_b, rate)
    ops.rglru_scan(o, ab, proj, 0, W, state, step, taps)
    lim = dict(rtol=1e-2, atol=6e-3) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=2e-5)
    for r, n in enumerate(lens):
        mine = proj[starts[r]:starts[r + 1]]
        want, S = plain_unit(mine, c, W, dtype if dtype == torch.bfloat16 else None)
        assert torch.allclose(o[starts[r]:starts[r + 1]].double().cpu(), want, **lim), r
        assert torch.allclose(state[slots[r], :W].double().cpu(), S, **lim), r
        alone = torch.zeros(1, 4 * W, device=DEV)
        cuts = [n] if n < 3 else [2, n - 2] if n < 20 else [n // 3, 2, n - n // 3 - 2]
        again, _ = run_unit(ops, mine, alone, c, cuts, [0], W, blocks, taps)
        assert close(again, o[starts[r]:starts[r + 1]], dtype, 1.0), r
    many = torch.randn(11 * 3, 2 * W, generator=g, device=DEV).to(dtype)
    state = torch.zeros(11, 4 * W, device=DEV)
    out, _ = run_unit(ops, many, state, c, [1, 1, 1], list(range(10, -1, -1)), W, blocks, taps)
    for r in range(11):
        want, _ = plain_unit(many[3 * r:3 * r + 3], c, W, dtype if dtype == torch.bfloat16 else None)
        assert torch.allclose(out[3 * r:3 * r + 3].double().cpu(), want, **lim), r


@DTYPES
def test_a_slow_channel_keeps_an_input_for_hundreds_of_tokens(ops, dtype):
    """One loud input, then silence: a channel with lam far below zero still holds its share 600 tokens later, in portions
    and one by one, a fast one has forgotten it; the addend keeps its digits where the decay is close to one."""
    W, taps = 16, 1
    c = SimpleNamespace(conv=torch.ones(W, 1, device=DEV), conv_b=torch.zeros(W, device=DEV),
                        ra=torch.zeros(2, 8, 8, dtype=dtype, device=DEV), ri=torch.zeros(2, 8, 8, dtype=dtype, device=DEV),
                        ra_b=torch.zeros(W, device=DEV), ri_b=torch.full((W,), 20.0, device=DEV),
                        lam=torch.linspace(-9.5, 1.0, W, device=DEV))
    T = 600
    proj = torch.zeros(T, 2 * W, dtype=dtype, device=DEV)
    proj[:, :W] = 3.0
    proj[0, W:] = 2.0
    want, S = plain_unit(proj, c, W)
    assert float(S[0]) > 0.01 and float(S[-1]) == 0.0
    for cuts in ([T], [2] * 300, [250, 300, 50], [1] * T):
        state = torch.zeros(1, W, device=DEV)
        run_unit(ops, proj, state, c, cuts, [0], W, 2, taps)
        assert torch.allclose(state[0].double().cpu(), S, rtol=2e-4, atol=1e-7), cuts[:2]


def test_gates_at_their_extremes(ops):
    """Decays of one and of nothing: no NaN, no lost digits (64-bit formulas), in both engine types."""
    for dtype in (torch.float32, torch.bfloat16):
        W = 64
        zr = torch.linspace(-40, 40, W, device=DEV)
        u = torch.ones(5, W, dtype=dtype, device=DEV)
        zero = torch.zeros(1, W, W, dtype=dtype, device=DEV)
        for rate in (1e-6, 1e-3, 0.2, 0.3, 3.0, 30.0):
            ab = torch.empty(5, W, 2, device=DEV)
            ops.rglru_gates(ab, u, zero, zero, zr, torch.full((W,), 3.0, device=DEV), torch.full((W,), rate, device=DEV))
            la = -torch.tensor(rate, dtype=torch.float32).double() * torch.sigmoid(zr.double().cpu())
            want = torch.sqrt(-torch.expm1(2 * la)) * torch.sigmoid(torch.tensor(3.0, dtype=torch.float64))
            assert torch.allclose(ab[0, :, 0].double().cpu(), torch.exp(la), rtol=3e-6, atol=1e-30)
            assert torch.allclose(ab[4, :, 1].double().cpu(), want, rtol=1e-5, atol=1e-12), (dtype, rate)


# -- experts by table, the clamped gated unit --------------------------------------------------------------------------------
def test_pairs_are_sorted_by_the_tables_experts(ops):
    g = torch.Generator().manual_seed(0)
    for T, top, E, vocab in ((1, 2, 5, 11), (37, 3, 7, 50), (700, 2, 12, 300), (5, 1, 1, 4)):
        table = torch.rand(vocab, E, generator=g).argsort(1)[:, :top].to(torch.int32)
        ids = torch.randint(0, vocab, (T,), generator=g).to(torch.int32)
        ids[0] = vocab - 1
        offsets, order, place, tiles = ops.moe_align(ids.to(DEV), E, table=table.to(DEV).contiguous())
        flat = table[ids.long()].reshape(-1)
        off = offsets[:E + 1].tolist()
        assert off == [0] + torch.bincount(flat.long(), minlength=E).cumsum(0).tolist()
        order, place = order[:T * top].cpu().long(), place[:T * top].cpu().long()
        assert torch.equal(order[place], torch.arange(T * top))
        for e in range(E):
            assert bool((flat[order[off[e]:off[e + 1]]] == e).all())


def clamped(gate, up, limit):
    g, u = torch.clamp(gate, max=limit), torch.clamp(up, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


@DTYPES
@pytest.mark.parametrize("T,inter", [(3, 24), (70, 33), (300, 256), (1, 1)])
def test_clamped_gated_unit_of_column_pairs(ops, dtype, T, inter):
    g = torch.Generator(device=DEV).manual_seed(inter)
    gu = (torch.randn(T, 2 * inter, generator=g, device=DEV) * 4).to(dtype)
    for limit in (0.5, 3.0, float("inf")):
        out = torch.empty(T, inter, dtype=dtype, device=DEV)
        ops.glu_pairs(out, gu, (limit, 1.702, 1.0))
        assert close(out, clamped(gu[:, 0::2].double(), gu[:, 1::2].double(), limit), dtype, 2.0)


def test_clamped_gated_unit_of_a_product_left_unreduced(ops):
    from turingserve_b200 import kernels
    g = torch.Generator(device=DEV).manual_seed(1)
    x = torch.randn(8, 1024, generator=g, device=DEV).to(torch.bfloat16)
    w = (torch.randn(192, 1024, generator=g, device=DEV) * 0.1).to(torch.bfloat16)
    gu = torch.empty(8, 192, dtype=torch.bfloat16, device=DEV)
    put_off = ops.linear(gu, x, w, may_defer=True)
    assert isinstance(put_off, kernels.LazyProduct)
    a, b = (torch.empty(8, 96, dtype=torch.bfloat16, device=DEV) for _ in range(2))
    ops.glu_pairs(a, put_off, (1.0, 1.702, 1.0))
    ops.glu_pairs(b, ops.linear(torch.empty_like(gu), x, w), (1.0, 1.702, 1.0))
    assert torch.equal(a, b)


def table_part(dtype, W, E, top, ff, limit, shared, vocab, seed, rank_scale=1.0):
    from turingserve_b200.config.model_config import RoutedMLPSpec
    from turingserve_b200.parts.base import BuildContext, build
    kw = dict(shared_intermediate_size=shared[0], shared_glu_limit=shared[1]) if shared else {}
    part = build("feed_forward", RoutedMLPSpec(
        num_experts=E, top_k=top, intermediate_size=ff, activation="clamped_glu", weight_on="output", gated=True, table_rows=vocab,
        glu_limit=limit, **kw), BuildContext(W, dtype, torch.device(DEV), 0))
    g = torch.Generator().manual_seed(seed)
    weights = {}
    for n, p in part.parameters().items():
        if p.integer:
            weights[n] = torch.rand(vocab, E, generator=g).argsort(1)[:, :top].to(torch.int32)
        else:
            weights[n] = (torch.randn(p.shape, generator=g) * 1.5 / math.sqrt(p.shape[1])).to(dtype)
    part.load({n: t.to(DEV) for n, t in weights.items()})
    ff_cfg = {"router": {"experts": E, "top": top}, "expert": {"limit": limit}}
    if shared:
        ff_cfg["shared"] = {"limit": shared[1]}
    return part, {n: (t.double() if t.dtype.is_floating_point else t) for n, t in weights.items()}, ff_cfg


@DTYPES
@pytest.mark.parametrize("T", [1, 4, 20, 90, 700])
@pytest.mark.parametrize("W,E,top,ff,limit,shared", [(72, 5, 2, 24, 0.8, (16, 0.5)), (64, 4, 4, 33, 1.5, None),
                                                     (128, 9, 3, 64, 0.9, (96, 0.3)), (40, 3, 1, 8, 0.6, (8, 2.0))])
def test_routed_experts_by_table(ops, dtype, T, W, E, top, ff, limit, shared):
    """The few-row, tiled and per-expert product paths, with group sizes read back and counted on the host; the rows left
    to the norm's kernel and the sum of its own."""
    vocab = 61
    part, weights, cfg = table_part(dtype, W, E, top, ff, limit, shared, vocab, W + top)
    ids = torch.randint(0, vocab, (T,), generator=torch.Generator().manual_seed(T))
    x = torch.randn(T, W, generator=torch.Generator(device=DEV).manual_seed(T), device=DEV).to(dtype)
    want = plain.table_moe(x.double().cpu(), ids, weights, "", cfg)
    for host in (None, ids.numpy()):
        step = SimpleNamespace(input_ids=ids.to(torch.int32).to(DEV), host_ids=host)
        got = part.forward(x, step)
        assert close(got, want, dtype, 3.0), float((got.double().cpu() - want).abs().max())
        pending = part.forward_pending(x, step)
        stream, out = torch.zeros(T, W, device=DEV), torch.empty(T, W, dtype=dtype, device=DEV)
        ops.post_norm(out, stream, pending.add, torch.ones(W, device=DEV), 1e-6, rows=pending.rows, place=pending.place,
                      top=pending.top, scale=pending.scale)
        assert close(stream, plain.unit_rms(want, 1e-6), dtype, 3.0)


def test_experts_depend_on_the_id_alone(ops):
    """Equal rows with different ids go to different experts, equal ids in different rows to the same ones."""
    part, weights, cfg = table_part(torch.float32, 32, 6, 2, 16, 1.0, None, 20, 3)
    x = torch.ones(20, 32, device=DEV)
    step = SimpleNamespace(input_ids=i32(list(range(20))), host_ids=None)
    got = part.forward(x, step)
    for a in range(20):
        for b in range(20):
            same = set(weights["table"][a].tolist()) == set(weights["table"][b].tolist())
            assert bool(torch.allclose(got[a], got[b], atol=1e-6)) == same
