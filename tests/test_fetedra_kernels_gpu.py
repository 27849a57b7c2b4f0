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
@pytest.mark.parametrize("T,N,R", [(1, 14, 5), (3, 192, 16), (70, 100, 33), (130, 256, 64), (2, 64, 1), (300, 320, 128), (65, 72, 24)])
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
