"""The kernels Fetedra brings, each alone against the plain functions: mixes of a token with its predecessor, the decay, the
recurrence with a state that fades channel by channel (whole, in portions, token by token, the one-kernel steps), the parts of a
latent attention (rows, queries, attention with window, sinks and gates, far keys and keys at every edge), grouped routing with
a correction, and the gated shared expert."""

from __future__ import annotations

import math
from types import SimpleNamespace

import pytest
import torch

from tests import plain_fetedra as plain

pytestmark = pytest.mark.gpu
DEV = "cuda"


@pytest.fixture(scope="module")
def ops():
    from turingserve_b200 import kernels
    kernels.use(None)
    return kernels.ops()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def close(got, want, dtype, slack=1.0):
    """Within ``slack`` roundings of a value one larger."""
    unit = (2.0 ** -8 if dtype == torch.bfloat16 else 2.0 ** -20) * slack
    d = (got.double().cpu() - want.double().cpu()).abs()
    return bool((d <= unit * (want.double().cpu().abs() + 1.0)).all())


DTYPES = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def batch(cuts, slots):
    """A step that brings cuts[b] tokens of the request in slots[b]."""
    starts = [0]
    for n in cuts:
        starts.append(starts[-1] + n)
    return SimpleNamespace(q_start=i32(starts), state_slots=i32(slots), num_requests=len(cuts), max_q_len=max(cuts),
                           token_request=i32([b for b, n in enumerate(cuts) for _ in range(n)]), num_tokens=starts[-1])


# -- the time mixer ------------------------------------------------------------------------------------------------------
@DTYPES
@pytest.mark.parametrize("hidden", [33, 60, 128, 2048, 1000])
def test_mixes_of_a_token_and_the_one_before(ops, dtype, hidden):
    """Portions of unequal requests: the row before a request's first token is its slot's, not its batch neighbour's."""
    g = torch.Generator(device=DEV).manual_seed(hidden)
    for cuts, slots in (([1, 1, 1], [2, 0, 3]), ([5, 1, 2, 9], [3, 1, 4, 0]), ([300], [2])):
        step = batch(cuts, slots)
        T, off = step.num_tokens, 8
        h = torch.randn(T, hidden, generator=g, device=DEV).to(dtype)
        mu = torch.randn(5, hidden, generator=g, device=DEV).to(dtype)
        state = torch.randn(5, -(-(off + hidden) // 4) * 4, generator=g, device=DEV)
        out = torch.empty(5, T, hidden, dtype=dtype, device=DEV)
        ops.token_shift(out, h, mu, state, off, step)
        at = 0
        for b, n in enumerate(cuts):
            rows = torch.cat([state[slots[b], off:off + hidden][None].double(), h[at:at + n].double()], 0)
            for i in range(5):
                want = plain.shifted_mix(rows, mu[i].double())[1:]
                assert close(out[i, at:at + n], want, dtype, 4.0), (b, i)
            at += n


@DTYPES
@pytest.mark.parametrize("T,N,R", [(1, 14, 5), (3, 200, 16), (70, 100, 33), (130, 256, 64), (2, 64, 1), (300, 320, 128), (65, 72, 24)])
def test_decays(ops, dtype, T, N, R):
    """From decays that keep everything to decays that keep nothing, all in 32-bit in both engine types."""
    g = torch.Generator(device=DEV).manual_seed(T + N)
    z = torch.randn(T, R, generator=g, device=DEV) * 2
    w2 = (torch.randn(N, R, generator=g, device=DEV) * 2 * R ** -0.5).to(dtype)
    w0 = torch.linspace(-18.0, 4.0, N, device=DEV)
    out = torch.empty(T, N, device=DEV)
    ops.wkv_decay(out, z, w2, w0)
    want = torch.exp(-torch.exp(torch.tanh(z.double()) @ w2.double().T + w0.double()))
    assert float((out.double() - want).abs().max()) < 2e-5


class Unit:
    """A time mixer's tensors and the plain answer for whole sequences."""

    def __init__(self, g, H, D, hidden, R, dtype, slow=False):
        rn = lambda *s: torch.randn(*s, generator=g, device=DEV)
        n = H * D
        self.H, self.D, self.hidden, self.R, self.n, self.dtype = H, D, hidden, R, n, dtype
        self.mu, self.w = (0.5 + 0.3 * rn(5, hidden)).to(dtype), (rn(4, n, hidden) * hidden ** -0.5).to(dtype)
        self.w1, self.w2 = (rn(R, hidden) * hidden ** -0.5).to(dtype), (rn(n, R) * 0.5 * R ** -0.5).to(dtype)
        self.w0 = rn(n) * 0.5 - (7.0 if slow else 2.5)
        self.u, self.norm, self.eps = rn(H, D), 1.0 + 0.3 * rn(n), 1e-5
        self.off = n * D
        self.slot = -(-(self.off + hidden) // 4) * 4

    def plain(self, h):
        """[T, n] in float64, from the mixes and projections rounded as the engine rounds them."""
        T, H, D = h.shape[0], self.H, self.D
        rnd = lambda x: x.to(self.dtype).double()
        m = [rnd(plain.shifted_mix(h.double(), self.mu[i].double())) for i in range(5)]
        r, k, v, gate = (rnd(m[i] @ self.w[i].double().T) for i in range(4))
        w = plain.decay_of(m[4], self.w1.double(), self.w2.double(), self.w0.double())
        heads = lambda x: x.view(T, H, D).cpu()
        o, S = plain.fading_state_scan(heads(r), heads(k), heads(v), heads(w), self.u.double().cpu())
        return plain.unit_rms(o, self.eps).reshape(T, self.n) * self.norm.double().cpu() * plain.silu(gate.cpu()), S

    def run(self, ops, h, step, state, one_kernel=True):
        T = h.shape[0]
        rkvg = torch.empty(4, T, self.n, dtype=self.dtype, device=DEV)
        z = torch.empty(T, self.R, device=DEV)
        used = [False, False]
        if one_kernel:
            used[0] = ops.wkv_project(rkvg, z, h, self.mu, self.w, self.w1, state, self.off, step)
        if not used[0]:
            mixes = torch.empty(5, T, self.hidden, dtype=self.dtype, device=DEV)
            ops.token_shift(mixes, h, self.mu, state, self.off, step)
            for i in range(4):
                ops.linear(rkvg[i], mixes[i], self.w[i])
            ops.linear(z, mixes[4], self.w1)
        y = torch.empty(T, self.n, dtype=self.dtype, device=DEV)
        if one_kernel:
            used[1] = ops.wkv_step(y, rkvg, z, self.w2, self.w0, self.u, self.norm, self.eps, h, state, step, self.H, self.D)
        if not used[1]:
            w, o = torch.empty(T, self.n, device=DEV), torch.empty(T, self.n, device=DEV)
            ops.wkv_decay(w, z, self.w2, self.w0)
            ops.wkv_scan(o, rkvg[0], rkvg[1], rkvg[2], w, self.u, h, state, step, self.H, self.D)
            ops.head_gated_rmsnorm(y, o, rkvg[3], self.norm, self.eps, self.H, self.D)
        return y, used


UNITS = pytest.mark.parametrize("H,D,hidden,R", [(3, 20, 60, 12), (2, 7, 33, 5), (4, 64, 128, 32), (2, 128, 96, 16), (1, 40, 48, 24),
                                                 (3, 48, 200, 16), (1, 256, 64, 8), (2, 33, 40, 1), (32, 64, 2048, 64)])


@DTYPES
@UNITS
def test_time_mixer_whole_in_portions_and_token_by_token(ops, dtype, H, D, hidden, R):
    """One sequence in four ways beside another request, slots that others left something in: the same outputs and the same
    last state, and the outputs are the plain ones."""
    g = torch.Generator(device=DEV).manual_seed(H * D)
    u = Unit(g, H, D, hidden, R, dtype)
    T = 37 if H * D <= 512 else 19
    h = torch.randn(T, hidden, generator=g, device=DEV).to(dtype)
    other = torch.randn(T + 8, hidden, generator=g, device=DEV).to(dtype)
    want, S = u.plain(h)
    slack = 4.0 if dtype == torch.bfloat16 else 60.0
    states = []
    for cuts in ([T], [2, 3, 16, T - 21] if T > 22 else [2, 3, T - 5], [1] * T, [T - 3, 1, 1, 1]):
        state = torch.randn(4, u.slot, generator=g, device=DEV)
        state[2].zero_()
        got, at = [], 0
        for n in cuts:
            rows, _ = u.run(ops, torch.cat([other[:n + 1], h[at:at + n]]), batch([n + 1, n], [0, 2]), state)
            got.append(rows[n + 1:])
            at += n
        out = torch.cat(got)
        assert close(out, want, dtype, slack), (cuts, float((out.double().cpu() - want).abs().max()))
        states.append(state[2].clone())
    assert close(states[0][:u.off].view(H, D, D), S, torch.float32, 2e4 if dtype == torch.bfloat16 else 60.0)
    lim = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=2e-2, atol=2e-2)
    for s in states:
        assert torch.equal(s[u.off:u.off + hidden], h[-1].float())
        assert torch.allclose(s[:u.off], states[0][:u.off], **lim)


@DTYPES
@UNITS
@pytest.mark.parametrize("B", [1, 5, 8, 9, 16, 20])
def test_single_tokens_in_one_kernel_steps(ops, dtype, H, D, hidden, R, B):
    """Batches of single tokens against the kernels of portions: products of 8 and of 16 rows, heads whose state one block holds
    and heads too wide for it; requests in slots of any order, other slots untouched."""
    g = torch.Generator(device=DEV).manual_seed(B)
    u = Unit(g, H, D, hidden, R, dtype)
    state = torch.randn(B + 2, u.slot, generator=g, device=DEV) * 0.3
    slots = torch.randperm(B + 2, generator=torch.Generator().manual_seed(B)).tolist()[:B]
    a, b = state.clone(), state.clone()
    for t in range(3):
        h = torch.randn(B, hidden, generator=g, device=DEV).to(dtype)
        step = batch([1] * B, slots)
        y1, used = u.run(ops, h, step, a)
        y2, _ = u.run(ops, h, step, b, one_kernel=False)
        assert used[0] == (dtype == torch.bfloat16 and hidden % 8 == 0 and B <= 16 and u.off % 4 == 0)
        assert used[1] == (-(-D // 32) * 32 * -(-D // 16) <= 1024)
        assert close(y1, y2, dtype, 4.0 if dtype == torch.bfloat16 else 60.0), (t, float((y1.float() - y2.float()).abs().max()))
    idle = [s for s in range(B + 2) if s not in slots]
    assert torch.equal(a[idle], state[idle]) and torch.equal(b[idle], state[idle])
    lim = dict(rtol=1e-5, atol=1e-5) if dtype == torch.float32 else dict(rtol=3e-2, atol=3e-2)
    assert torch.allclose(a[slots], b[slots], **lim)


@DTYPES
@pytest.mark.parametrize("D", [16, 20, 64, 100])
def test_a_slow_channel_keeps_a_value_for_a_thousand_tokens(ops, dtype, D):
    """One loud key and value, then silence: the read-out a thousand tokens later is the product of the decays between, in one
    portion, in portions and over single tokens; the bonus counts at the token itself only."""
    H, T = 1, 1000
    u = Unit(torch.Generator(device=DEV).manual_seed(3), H, D, 24, 4, dtype)
    r, k, v = (torch.zeros(T, D, dtype=dtype, device=DEV) for _ in range(3))
    k[0, 5], v[0, 9] = 2.0, 3.0
    r[:, 5] = 1.0
    w = torch.rand(T, D, generator=torch.Generator(device=DEV).manual_seed(4), device=DEV) * 1e-3 + 0.9985
    bonus = torch.full((1, D), -0.5, device=DEV)
    h = torch.randn(T, 24, device=DEV).to(dtype)
    want = torch.zeros(T, dtype=torch.float64)
    want[0] = -3.0
    want[1:] = 6.0 * torch.cat([torch.ones(1, dtype=torch.float64), w[1:-1, 5].double().cpu().cumprod(0)])
    for cuts in ([T], [7, 16, 2, 1, 300, T - 326], [500] + [1] * 500):
        state, out, at = torch.zeros(1, u.slot, device=DEV), torch.empty(T, D, device=DEV), 0
        for n in cuts:
            s = slice(at, at + n)
            ops.wkv_scan(out[s], r[s], k[s], v[s], w[s], bonus, h[s], state, batch([n], [0]), H, D)
            at += n
        assert float((out[:, 9].double().cpu() - want).abs().max()) < 2e-4
        assert float(out[:, :9].abs().max()) == 0.0 and float(out[:, 10:].abs().max()) == 0.0


@DTYPES
@pytest.mark.parametrize("H,D", [(3, 24), (2, 64), (1, 128)])
def test_unequal_requests_in_one_scan_are_bit_for_bit_those_alone(ops, dtype, H, D):
    """Requests of 1 to 150 tokens in one launch, each alone, and each cut in two: the same bits of outputs and states."""
    g = torch.Generator(device=DEV).manual_seed(8)
    rn = lambda *s: torch.randn(*s, generator=g, device=DEV)
    cuts, slots, n, hid = [1, 150, 16, 17, 2, 33], [5, 0, 3, 1, 6, 2], H * D, 40
    T = sum(cuts)
    r, k, v = (rn(T, n).to(dtype) for _ in range(3))
    w, bonus, h = torch.rand(T, n, generator=g, device=DEV), rn(H, D), rn(T, hid).to(dtype)
    state = rn(7, n * D + hid)
    both, out = state.clone(), torch.empty(T, n, device=DEV)
    ops.wkv_scan(out, r, k, v, w, bonus, h, both, batch(cuts, slots), H, D)
    at = 0
    for m, slot in zip(cuts, slots):
        for parts in ([m], [m - m // 3, m // 3] if m > 2 else [m]):
            one, got, p = state.clone(), torch.empty(m, n, device=DEV), 0
            for q in parts:
                s, d = slice(at + p, at + p + q), slice(p, p + q)
                ops.wkv_scan(got[d], r[s], k[s], v[s], w[s], bonus, h[s], one, batch([q], [slot]), H, D)
                p += q
            assert torch.equal(got, out[at:at + m]) and torch.equal(one[slot], both[slot])
        at += m


@DTYPES
def test_norm_of_heads_with_weights_of_their_own(ops, dtype):
    g = torch.Generator(device=DEV).manual_seed(1)
    for T, H, V in ((9, 4, 15), (600, 5, 64), (3, 24, 64), (520, 3, 128)):
        x, gate = torch.randn(T, H * V, generator=g, device=DEV) * 3, torch.randn(T, H * V, generator=g, device=DEV).to(dtype)
        w = torch.randn(H * V, generator=g, device=DEV)
        out = torch.empty(T, H * V, dtype=dtype, device=DEV)
        ops.head_gated_rmsnorm(out, x, gate, w, 0.2, H, V)
        unit = plain.unit_rms(x.double().view(T, H, V), 0.2).reshape(T, H * V)
        assert close(out, unit * w.double() * plain.silu(gate.double()), dtype, 6.0)
        common = w[:V].contiguous()
        ops.head_gated_rmsnorm(out, x, gate, common, 0.2, H, V)
        assert close(out, unit * common.double().repeat(H) * plain.silu(gate.double()), dtype, 6.0)


# -- latent attention ----------------------------------------------------------------------------------------------------------
def freqs(base, dims):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], device=DEV)


def turn(x, pos, base, dims, pairing):
    if pairing == "halves":
        return plain.rotate_halves(x, pos, base, dims)
    order = list(range(0, dims, 2)) + list(range(1, dims, 2)) + list(range(dims, x.shape[-1]))     # neighbours -> halves
    y = plain.rotate_halves(x[..., order], pos, base, dims)
    back = torch.empty_like(y)
    back[..., order] = y
    return back


@DTYPES
@pytest.mark.parametrize("pairing", ["halves", "neighbours"])
@pytest.mark.parametrize("T,q_rank,rank,R,rot,extra", [(1, 20, 28, 6, 6, 3), (9, 14, 18, 10, 6, 5), (40, 768, 512, 64, 64, 12), (3, 8, 24, 4, 4, 0)])
def test_rows_of_a_latent_projection(ops, dtype, pairing, T, q_rank, rank, R, rot, extra):
    """The cached row and the query latent of every token; a slot of -1 caches nothing; other rows of the pool untouched."""
    g = torch.Generator(device=DEV).manual_seed(T + rank)
    n_in, page = q_rank + rank + R + extra, 8
    proj = (torch.randn(T, n_in, generator=g, device=DEV) * 2).to(dtype)
    kw, qw = 1 + 0.3 * torch.randn(rank, generator=g, device=DEV), 1 + 0.3 * torch.randn(q_rank, generator=g, device=DEV)
    pos = torch.randint(0, 3000, (T,), generator=g, device=DEV, dtype=torch.int32)
    slots = (torch.randperm(T + 16, generator=torch.Generator().manual_seed(T))[:T] + page).to(torch.int32).to(DEV)
    if T > 2:
        slots[1] = -1
    pool = torch.full((-(-(T + 16) // page) + 2, 1, page, rank + R), 7.0, dtype=dtype, device=DEV)
    cq = torch.empty(T, q_rank, dtype=dtype, device=DEV)
    back = ops.latent_kv_write(proj, q_rank, kw, 0.1, pos, freqs(50.0, rot), 1.0, rot, pool, slots, rank, R, page, pairing, cq, qw)
    assert back is proj
    p = proj.double().cpu()
    assert close(cq, plain.unit_rms(p[:, :q_rank], 0.1) * qw.double().cpu(), dtype, 4.0)
    c = plain.unit_rms(p[:, q_rank:q_rank + rank], 0.1) * kw.double().cpu()
    kr = turn(p[:, q_rank + rank:q_rank + rank + R], pos.cpu(), 50.0, rot, pairing)
    flat, seen = pool.view(-1, rank + R), []
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            seen.append(s)
            assert close(flat[s, :rank], c[t], dtype, 4.0)
            assert float((flat[s, rank:].double().cpu() - kr[t]).abs().max()) < (0.06 if dtype == torch.bfloat16 else 5e-3)
    rest = [i for i in range(flat.shape[0]) if i not in seen]
    assert bool((flat[rest] == 7.0).all())


@pytest.mark.parametrize("T", [1, 8, 40])
def test_rows_of_a_product_left_unreduced(ops, T):
    """The projection's partial sums: the values from the finished product, gates finished in place."""
    from turingserve_b200 import kernels
    g = torch.Generator(device=DEV).manual_seed(T)
    q_rank, rank, R, H, K, page = 96, 64, 16, 6, 1024, 16
    n_in = q_rank + rank + R + 8
    x = torch.randn(T, K, generator=g, device=DEV).to(torch.bfloat16)
    w = (torch.randn(n_in, K, generator=g, device=DEV) * 0.05).to(torch.bfloat16)
    kw, qw = torch.ones(rank, device=DEV), torch.ones(q_rank, device=DEV)
    pos, slots = i32(list(range(T))), i32(list(range(page, page + T)))
    results = []
    for defer in (False, True):
        proj = torch.empty(T, n_in, dtype=torch.bfloat16, device=DEV)
        p = ops.linear(proj, x, w, may_defer=defer, lazy=False)
        assert isinstance(p, kernels.Deferred) == defer
        pool = torch.zeros(8, 1, page, rank + R, dtype=torch.bfloat16, device=DEV)
        cq = torch.empty(T, q_rank, dtype=torch.bfloat16, device=DEV)
        back = ops.latent_kv_write(p, q_rank, kw, 1e-6, pos, freqs(100.0, R), 1.0, R, pool, slots, rank, R, page, "halves", cq, qw,
                                   (q_rank + rank + R, H))
        results.append((pool, cq, back[:, q_rank + rank + R:q_rank + rank + R + H].clone()))
    for a, b in zip(*results):
        assert close(a, b, torch.bfloat16, 2.0) and float(a.abs().max()) > 0


@DTYPES
@pytest.mark.parametrize("pairing", ["halves", "neighbours"])
@pytest.mark.parametrize("T", [1, 7, 8, 13, 16, 17, 70])
@pytest.mark.parametrize("H,N,K,R,rot", [(3, 28, 10, 6, 6), (3, 256, 32, 64, 64), (12, 512, 128, 64, 64), (2, 96, 320, 8, 4), (5, 72, 24, 16, 16)])
def test_queries_into_the_latent_space(ops, dtype, pairing, T, H, N, K, R, rot):
    g = torch.Generator(device=DEV).manual_seed(T * H)
    q = torch.randn(T, H * (K + R), generator=g, device=DEV).to(dtype)
    w = (torch.randn(H, N, K, generator=g, device=DEV) * K ** -0.5).to(dtype)
    pos = torch.randint(0, 2000, (T,), generator=g, device=DEV, dtype=torch.int32)
    qa = torch.empty(T, H, N + R, dtype=dtype, device=DEV)
    ops.latent_queries(qa, q, w, pos, freqs(80.0, rot), 1.0, rot, pairing)
    heads = q.double().cpu().view(T, H, K + R)
    assert close(qa[:, :, :N], torch.einsum("thk,hnk->thn", heads[:, :, :K], w.double().cpu()), dtype, 8.0)
    want = turn(heads[:, :, K:], pos.cpu(), 80.0, rot, pairing)
    assert float((qa[:, :, N:].double().cpu() - want).abs().max()) < (0.04 if dtype == torch.bfloat16 else 3e-3)


@pytest.mark.parametrize("T", [1, 8, 9, 16, 24])
def test_queries_of_a_product_left_unreduced(ops, T):
    from turingserve_b200 import kernels
    g = torch.Generator(device=DEV).manual_seed(T)
    H, N, K, R, rank = 4, 128, 64, 32, 512
    x = torch.randn(T, rank, generator=g, device=DEV).to(torch.bfloat16)
    uq = (torch.randn(H * (K + R), rank, generator=g, device=DEV) * 0.05).to(torch.bfloat16)
    w = (torch.randn(H, N, K, generator=g, device=DEV) * 0.1).to(torch.bfloat16)
    pos, out = i32(list(range(5, 5 + T))), []
    for defer in (False, True):
        q = ops.linear(torch.empty(T, H * (K + R), dtype=torch.bfloat16, device=DEV), x, uq, may_defer=defer, lazy=False)
        assert isinstance(q, kernels.Deferred) == defer
        qa = torch.empty(T, H, N + R, dtype=torch.bfloat16, device=DEV)
        ops.latent_queries(qa, q, w, pos, freqs(80.0, R), 1.0, R, "halves")
        out.append(qa)
    assert close(out[0], out[1], torch.bfloat16, 2.0) and float(out[0].abs().max()) > 0


@pytest.mark.parametrize("T", [1, 8, 11, 16])
@pytest.mark.parametrize("H,N,K", [(12, 128, 512), (3, 40, 256), (2, 9, 1032), (5, 33, 8)])
def test_products_per_head_of_few_rows(ops, T, H, N, K):
    """Strided rows in and out, the tensor-core instances with k whole and in four shares."""
    g = torch.Generator(device=DEV).manual_seed(N)
    x = torch.randn(T, H, K + 8, generator=g, device=DEV).to(torch.bfloat16)[:, :, :K]
    w = (torch.randn(H, N, K, generator=g, device=DEV) * K ** -0.5).to(torch.bfloat16)
    wide = torch.full((T, H, N + 2), 5.0, dtype=torch.bfloat16, device=DEV)
    ops.batched_linear(wide[:, :, :N], x, w)
    assert close(wide[:, :, :N], torch.einsum("thk,hnk->thn", x.double().cpu(), w.double().cpu()), torch.bfloat16, 8.0)
    assert bool((wide[:, :, N:] == 5.0).all())


def run_attention(ops, q, rows, q_lens, page, rank, scale, window, sinks, gate):
    """q [T, H, row]; rows: every request's cached rows up to its length; pages in a shuffled pool, those a window has passed
    for every query given back (their entries name the null page)."""
    rng = torch.Generator().manual_seed(len(rows))
    n_pages = [-(-r.shape[0] // page) for r in rows]
    order = (torch.randperm(sum(n_pages), generator=rng) + 1).tolist()
    pool = torch.zeros(sum(n_pages) + 1, 1, page, q.shape[2], dtype=q.dtype, device=DEV)
    bt = torch.zeros(len(rows), max(n_pages), dtype=torch.int32)
    at, starts = 0, [0]
    for r, (x, n) in enumerate(zip(rows, n_pages)):
        mine = order[at:at + n]
        at += n
        bt[r, :n] = torch.tensor(mine)
        for p, place in enumerate(mine):
            part = x[p * page:(p + 1) * page]
            pool[place, 0, :part.shape[0]] = part
        if window:
            bt[r, :max(0, x.shape[0] - q_lens[r] - window + 1) // page] = 0
        starts.append(starts[-1] + q_lens[r])
    lens = [x.shape[0] for x in rows]
    step = SimpleNamespace(q_start=i32(starts), seq_lens=i32(lens), num_requests=len(rows), num_decode=sum(1 for n in q_lens if n == 1),
                           max_q_len=max(q_lens), max_seq_len=max(lens))
    out = torch.empty(q.shape[0], q.shape[1], rank, dtype=q.dtype, device=DEV)
    ops.attention_biased(out, q, pool, None, bt.to(DEV), step, 1, page, scale, 0.0, None, window, sinks=sinks, gate=gate)
    return out


def plain_attention(q, rows, rank, scale, window, sinks, gate):
    T, n, H = rows.shape[0], q.shape[0], q.shape[1]
    ok = plain.visible(T, window)[T - n:]
    k = rows.double().cpu()
    out = []
    for h in range(H):
        p = plain.sink_softmax(q[:, h].double().cpu() @ k.T * scale, ok, sinks[h].double().cpu())
        out.append(p @ k[:, :rank] * torch.sigmoid(gate[:, h].double().cpu())[:, None])
    return torch.stack(out, 1)


# (rank, rotated width): rows the tensor-core instances take (bfloat16) and others
ROWS = pytest.mark.parametrize("dtype,H,rank,R,page", [
    (torch.float32, 3, 28, 6, 16), (torch.bfloat16, 3, 28, 6, 16), (torch.bfloat16, 5, 96, 24, 64), (torch.bfloat16, 12, 256, 64, 64),
    (torch.bfloat16, 28, 512, 64, 64), (torch.bfloat16, 40, 256, 64, 16), (torch.float32, 6, 256, 64, 64), (torch.bfloat16, 2, 512, 64, 8)])


@ROWS
@pytest.mark.parametrize("window", [None, 1, 30, 64, 100])
@pytest.mark.parametrize("splits", [0, 3])
def test_attention_in_batches_of_unequal_requests(ops, dtype, H, rank, R, page, window, splits):
    """Single tokens and portions in one launch, windows that end inside, at and past tiles, sinks, gates in columns of a wider
    tensor, pages that the window has passed given back."""
    g = torch.Generator(device=DEV).manual_seed(H * rank + (window or 0))
    q_lens, lens = [1, 1, 1, 1, 2, 40, 7], [1, 64, 333, 129, 71, 150, 7]
    T, row = sum(q_lens), rank + R
    q = (torch.randn(T, H, row, generator=g, device=DEV) * 1.5).to(dtype)
    rows = [torch.randn(n, row, generator=g, device=DEV).to(dtype) for n in lens]
    gate = torch.randn(T, H + 16, generator=g, device=DEV).to(dtype)[:, 8:8 + H]
    sinks = torch.randn(H, generator=g, device=DEV) + 1.0
    old = ops.biased_decode_splits
    ops.biased_decode_splits = splits
    try:
        got = run_attention(ops, q, rows, q_lens, page, rank, row ** -0.5, window, sinks, gate)
    finally:
        ops.biased_decode_splits = old
    at = 0
    for r, n in enumerate(q_lens):
        want = plain_attention(q[at:at + n], rows[r], rank, row ** -0.5, window, sinks, gate[at:at + n])
        assert close(got[at:at + n], want, dtype, 4.0 if dtype == torch.bfloat16 else 30.0), (r, float((got[at:at + n].double().cpu() - want).abs().max()))
        at += n


@pytest.mark.parametrize("decode", [False, True])
@ROWS
def test_one_loud_key_at_every_edge(ops, decode, dtype, H, rank, R, page):
    """Every key is silent but one, whose value is marked: the query finds it exactly where the window lets it, just inside and
    just outside, at page borders, far away, and never ahead of itself; a sink takes half of what equals it."""
    row, marked = rank + R, 3
    sinks, gate_row = torch.full((H,), 20.0, device=DEV), 30.0
    for T, window in ((330, 100), (150, 64), (321, 1), (90, 200), (700, None)):
        n_q = 1 if decode else 24
        i, w = T - 1, window or T
        places = {i, i - 1, i - w + 1, i - w, i - w - 1, 0, 1, page - 1, page, (i // page) * page, (i // page) * page - 1, i // 2}
        for j in sorted(p for p in places if 0 <= p <= i):
            k = torch.zeros(T, row, dtype=dtype, device=DEV)
            k[j, rank + 1] = 20.0
            k[j, marked] = 1.0
            q = torch.zeros(n_q, H, row, dtype=dtype, device=DEV)
            q[:, :, rank + 1] = 1.0
            gate = torch.full((n_q, H), gate_row, dtype=dtype, device=DEV)
            out = run_attention(ops, q, [k], [n_q], page, rank, 1.0, window, sinks, gate)[:, H - 1, marked].tolist()
            for at, value in enumerate(out):
                p = T - n_q + at
                seen = j <= p and p - j < w
                assert abs(value - (0.5 if seen else 0.0)) < 1e-3, (T, window, j, p, value)


# -- routing ------------------------------------------------------------------------------------------------------------------
@DTYPES
@pytest.mark.parametrize("E,top,groups,keep", [(20, 2, 2, 1), (12, 3, 4, 2), (6, 2, 6, 3), (9, 1, 3, 1), (5, 2, 1, 1), (64, 6, 8, 3), (8, 4, 2, 2),
                                               (130, 5, 65, 7)])
def test_grouped_routing(ops, dtype, E, top, groups, keep):
    """Choices by scores with corrections (negative ones too), groups by their two largest; weights without the correction over
    their sum, times a constant; the shared expert's weight beside them."""
    g = torch.Generator(device=DEV).manual_seed(E + top)
    T, K = 50, 72
    x = torch.randn(T, K, generator=g, device=DEV).to(dtype)
    w = torch.randn(E + 1, K, generator=g, device=DEV) * 0.2
    corr = torch.randn(E, generator=g, device=DEV) * 0.3 - 0.6
    idx, wts, share = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV), torch.empty(T, device=DEV)
    ops.router_topk(idx, wts, x, w, False, True, corr, groups, keep, 1.7, share)
    s = torch.sigmoid(x.double().cpu() @ w.double().cpu().T)
    assert float((share.double().cpu() - s[:, E]).abs().max()) < 1e-5
    assert bool((s[:, :E] + corr.double().cpu() < 0).any())
    right = 0
    for t in range(T):
        want = plain.choose(s[t, :E], corr.double().cpu(), top, groups, keep)
        got = idx[t].tolist()
        if got != want:                              # (two choice scores or two groups closer than 32-bit arithmetic tells apart)
            continue
        right += 1
        picked = s[t, got]
        assert float((wts[t].double().cpu() - picked / picked.sum() * 1.7).abs().max()) < 1e-5
    assert right >= T - 1


def test_a_kept_group_without_the_best_expert(ops):
    """The single best expert lies in a group whose two largest add up to less: it must not be chosen; without a correction
    vector the groups go by the scores."""
    logit = lambda p: math.log(p / (1 - p))
    scores = [0.95, 0.05, 0.1, 0.6, 0.7, 0.2]                      # groups of three: 0.95 + 0.1 against 0.7 + 0.6
    w = torch.tensor([[logit(p)] for p in scores], device=DEV)
    x = torch.ones(1, 1, device=DEV)
    idx, wts = torch.empty(1, 2, dtype=torch.int32, device=DEV), torch.empty(1, 2, device=DEV)
    ops.router_topk(idx, wts, x, w, False, True, None, 2, 1)
    assert idx[0].tolist() == [4, 3] and torch.allclose(wts[0], torch.tensor([0.7, 0.6], device=DEV) / 1.3, atol=1e-6)
    ops.router_topk(idx, wts, x, w, False, False, None, 2, 2, 3.0)
    assert idx[0].tolist() == [0, 4] and torch.allclose(wts[0], torch.tensor([2.85, 2.1], device=DEV), atol=1e-5)


@DTYPES
@pytest.mark.parametrize("T", [1, 5, 30, 400])
@pytest.mark.parametrize("W,E,top,ff,groups,shared", [(72, 12, 3, 24, (4, 2), (16, 0.5)), (64, 4, 4, 33, (1, 1), None), (128, 16, 2, 64, (8, 3), (96, 0.9))])
def test_routed_feed_forward(ops, dtype, T, W, E, top, ff, groups, shared):
    """The whole part against the plain one; many rows go to products of the experts' own."""
    from turingserve_b200.config.model_config import RoutedMLPSpec
    from turingserve_b200.parts.base import BuildContext, build
    kw = dict(shared_intermediate_size=shared[0], shared_glu_limit=shared[1], shared_gate=True) if shared else {}
    spec = RoutedMLPSpec(num_experts=E, top_k=top, intermediate_size=ff, activation="clamped_glu", gated=True, scoring="sigmoid", renormalize=True,
                         weight_on="output", correction=True, groups=groups[0], groups_kept=groups[1], weight_scale=1.4, glu_limit=0.8, **kw)
    part = build("feed_forward", spec, BuildContext(W, dtype, torch.device(DEV), 0))
    g = torch.Generator(device=DEV).manual_seed(W)
    t = {n: torch.randn(p.shape, generator=g, device=DEV) * (2.0 * p.shape[-1] ** -0.5) for n, p in part.parameters().items()}
    t["correction"] = torch.randn(E, generator=g, device=DEV) * 0.2 - 0.5
    t = {n: v.to(dtype) if part.parameters()[n].compute_dtype else v for n, v in t.items()}
    part.load(t)
    x = torch.randn(T, W, generator=g, device=DEV).to(dtype)
    got = part.forward(x)
    f = {"router": {"top": top, "scale": 1.4, "groups": {"count": groups[0], "keep": groups[1]}}, "expert": {"limit": 0.8},
         "shared": {"limit": shared[1]} if shared else None}
    want = plain.routed_ff(x.double().cpu(), {n: v.double().cpu() for n, v in t.items()}, "", f)
    err = (got.double().cpu() - want).abs().amax(1)
    bad = int((err > (0.03 if dtype == torch.bfloat16 else 1e-5) * float(want.abs().max())).sum())
    assert bad <= T // 100, (bad, float(err.max()))                 # (two choice scores closer than 32-bit arithmetic tells apart)
