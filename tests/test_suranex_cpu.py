"""Suranex without a GPU: the parser and its refusals, checkpoint names, the memory the two mixers declare (pages whose
first ones a window keeps, one flat state slot), tables of experts, the engine's host logic (portions down to two tokens,
mixed batches, pages and slots used again) through the kernel twins against the plain model, and the plain model's
mechanisms against closed forms."""

from __future__ import annotations

import json
import math

import pytest
import torch

from tests import plain_suranex as plain
from tests import schedules
from tests import suranex_tiny as st
from turingserve_b200.cache.manager import CacheManager, RunNeeds
from turingserve_b200.config.model_config import NormedAttentionSpec, RGLRUSpec, RoutedMLPSpec, YarnRotarySpec
from turingserve_b200.config.registry import get_architecture, load_model_config
from turingserve_b200.parts.base import BuildContext, CacheNeed, ParamSpec, StateNeed, build


def test_parser_reads_every_size_and_option():
    cfg = st.tiny_config("A")
    assert cfg.architecture == "Suranex" and (cfg.hidden_size, cfg.vocab_size) == (72, 131) and not cfg.tie_word_embeddings
    assert [r.layer for r in cfg.schedule] == [0, 1, 2, 3] and cfg.final_norm.eps == 1e-5 and cfg.final_norm.weight_offset == 1.0
    a = cfg.layers[0].mixer
    assert a == NormedAttentionSpec(
        num_heads=4, num_kv_heads=2, key_dim=16, value_dim=8, scale=0.4, norm_eps=1e-5, softcap=5.0, window=7, keep_first=3,
        position=YarnRotarySpec(base=100.0, dims=8, factor=8.0, original=40.0, fast=4.0, slow=1.0, pairing="halves"),
        value_base=100.0)
    assert cfg.layers[1].mixer == RGLRUSpec(width=60, num_blocks=3, conv_taps=4)
    f = cfg.layers[1].feed_forward
    assert isinstance(f, RoutedMLPSpec) and (f.num_experts, f.top_k, f.intermediate_size, f.shared_intermediate_size) == (5, 2, 24, 40)
    assert (f.glu_limit, f.shared_glu_limit, f.glu_slope, f.glu_offset, f.table_rows) == (0.6, 1.1, 1.702, 1.0, 131)
    assert "feed_forward" not in cfg.layers[2].roles and cfg.layers[3].feed_forward.shared_intermediate_size is None
    b = st.tiny_config("B")
    m = b.layers[2].mixer
    assert m.position is None and m.value_base is None and m.window is None and m.keep_first == 0 and m.softcap == 3.0
    assert b.layers[1].mixer.softcap is None and b.layers[1].mixer.window == 40 and b.layers[1].mixer.keep_first == 0
    assert b.layers[1].feed_forward.glu_limit == float("inf")


def test_names_round_trip_and_registry(tmp_path):
    for name in st.TINY:
        cfg = st.tiny_config(name)
        arch = get_architecture("Suranex")
        again = arch.parse_config(json.loads(json.dumps(arch.to_config_json(cfg))))
        assert again == cfg
        folder = st.make_tiny_folder(name, tmp_path)
        assert load_model_config(folder) == cfg
    names = set(arch.build_model(st.tiny_config("A"), torch.float32, "cpu", 1).parameters(arch.tensor_names(st.tiny_config("A"))))
    assert {"embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.q", "l0.mix.k", "l0.mix.v", "l0.mix.o", "l0.mix.g",
            "l0.mix.q.norm", "l0.mix.k.norm", "l0.mlp.table", "l0.mlp.e4.gate", "l0.mlp.e4.up", "l0.mlp.e4.down",
            "l0.mlp.shared.gate", "l0.mlp.shared.up", "l0.mlp.shared.down", "l1.mix.y", "l1.mix.y.b", "l1.mix.x", "l1.mix.x.b",
            "l1.mix.conv", "l1.mix.conv.b", "l1.mix.ra", "l1.mix.ra.b", "l1.mix.ri", "l1.mix.ri.b", "l1.mix.lam", "l1.mix.o"} <= names
    assert "l2.norm2" not in names and "l3.mlp.shared.up" not in names


def test_parser_refusals():
    ok = st.TINY["D"][0]

    def refused(change, text):
        layers = json.loads(json.dumps(ok["layers"]))
        change(layers)
        with pytest.raises(ValueError, match=text):
            cfg = st.make_config(**{**ok, "layers": layers})
            get_architecture("Suranex").build_model(cfg, torch.float32, "cpu", 1)

    refused(lambda l: l[0].update(type="conv"), "unknown layer type")
    refused(lambda l: l[0]["mlp"].update(kind="dense"), "unknown feed-forward")
    refused(lambda l: l[0]["mixer"].pop("scale"), "scale")
    refused(lambda l: l[0]["mixer"]["mask"].pop("size"), "size")
    refused(lambda l: l[0]["mixer"].update(vdim=9), "do not pair")
    refused(lambda l: l[0]["mixer"].update(kv_heads=3), "multiple")
    refused(lambda l: l[0]["mixer"]["rot"].update(dims=14), "rotated dimensions")
    refused(lambda l: l[1]["mixer"].update(blocks=7), "equal parts")
    refused(lambda l: l[1]["mixer"].update(conv=9), "taps")
    refused(lambda l: l[0]["mlp"]["router"].update(top=5), "top 5 of 4")


def test_memory_of_every_run():
    from turingserve_b200.engine.runner import run_needs
    model = get_architecture("Suranex").build_model(st.tiny_config("A"), torch.float32, "cpu", 1)
    needs = run_needs(model)
    assert needs[0].cache == CacheNeed(2, 16, 7, value_dim=8, keep_first=3) and needs[0].state is None
    assert needs[1].cache is None and needs[1].state == StateNeed((60 * 5,), torch.float32)
    assert needs[2].cache == CacheNeed(1, 10, 21, value_dim=14, keep_first=18)
    one_tap = get_architecture("Suranex").build_model(st.tiny_config("B"), torch.float32, "cpu", 1)
    assert run_needs(one_tap)[0].state == StateNeed((36,), torch.float32)


def test_a_window_keeps_the_pages_of_the_first_tokens():
    """Pages of 4: a window of 6 that keeps 5 first tokens holds pages 0 and 1 for good and gives the rest back as the
    window passes; the same window without kept tokens gives all back; needs that differ in kept tokens are two groups."""
    cm = CacheManager([RunNeeds(CacheNeed(1, 2, 6, keep_first=5), None), RunNeeds(CacheNeed(1, 2, 6), None)], 4, 30, 2)
    assert len(cm.groups) == 2
    rc = cm.admit("a")
    for n in range(1, 60):
        cm.grow(rc, 1)
        cm.advance(rc, 1)
        cm.check()
        kept, plain_ = rc.tables
        assert all(kept[p] for p in range(min(2, len(kept))))
        first = max(0, n - 6 + 1) // 4                     # the first page the next position's window needs
        assert [bool(p) for p in plain_] == [p >= first for p in range(len(plain_))]
        assert [bool(p) for p in kept] == [p < 2 or p >= first for p in range(len(kept))]
    cm.release(rc)
    cm.check()
    assert cm.min_free() == 29


def test_the_frequencies_of_the_product_are_the_plain_ones():
    ctx = BuildContext(8, torch.float32, torch.device("cpu"), 0)
    for base, dims, sc in ((100.0, 8, (8.0, 40.0, 4.0, 1.0)), (20000.0, 48, (4.0, 1500.0, 24.0, 1.0)), (30.0, 12, None),
                           (500000.0, 128, (16.0, 8192.0, 32.0, 2.0)), (50.0, 2, (2.0, 10.0, 1.0, 1.0))):
        scaling = dict(zip(("factor", "original", "fast", "slow"), sc)) if sc else None
        want, mag = plain.key_frequencies(base, dims, scaling)
        enc = build("position", YarnRotarySpec(base=base, dims=dims, pairing="halves", **(scaling or {})), ctx)
        assert enc.pairing == "halves" and torch.allclose(enc.freq.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6)
        assert abs(enc.magnitude - mag) < 1e-12


def test_random_tables_hold_different_experts_and_bad_tables_are_refused():
    from turingserve_b200.weights.random_init import random_tensors
    t = random_tensors(st.tiny_config("A"), 3)["l0.mlp.table"]
    assert t.dtype == torch.int32 and tuple(t.shape) == (131, 2) and int(t.min()) >= 0 and int(t.max()) == 4
    assert bool((t[:, 0] != t[:, 1]).all()) and len(set(map(tuple, t.tolist()))) > 10
    spec = RoutedMLPSpec(num_experts=3, top_k=2, intermediate_size=4, activation="clamped_glu", gated=True, weight_on="output",
                         table_rows=5)
    part = build("feed_forward", spec, BuildContext(6, torch.float32, torch.device("cpu"), 0))
    assert part.parameters()["table"] == ParamSpec((5, 2), integer=True, init="distinct", high=3)
    tensors = {n: torch.zeros(p.shape, dtype=torch.int32 if p.integer else torch.float32) for n, p in part.parameters().items()}
    tensors["table"][4, 1] = 3
    with pytest.raises(ValueError, match="table names experts"):
        part.load(tensors)


def _replay_cpu(folder, name, steps, page=None):
    from turingserve_b200 import kernels
    from turingserve_b200.engine.replay import Replayer
    from tests.twin_ops import TwinOps
    kernels.use(TwinOps())
    try:
        rp = Replayer(folder, torch.float32, schedules.peak_tokens(steps), "cpu", page_size=page or st.page_size(name))
        outs = {}
        with torch.inference_mode():
            for s in steps:
                o = rp.step(s)
                if o is not None:
                    outs[s["step"]] = o
                rp.cache.check()
        assert not rp.cache.live
    finally:
        kernels.use(None)
    return schedules.collect(steps, outs)


@pytest.mark.parametrize("name", ["A", "B", "D"])
@pytest.mark.parametrize("schedule", ["decode_tail", "portions", "mixed"])
def test_host_logic_against_plain(tmp_path, name, schedule):
    """More requests than live slots, a pool that makes pages go round, state slots handed on from request to request,
    portions down to two tokens (shorter than the filter's memory) that end in the middle of pages and windows."""
    folder = st.make_tiny_folder(name, tmp_path)
    cfg, w = plain.read_folder(folder)
    reqs = {f"r{i}": st.random_ids(n, cfg["vocab"], 50 + i) for i, n in enumerate([1, 9, 34, 21, 17, 40])}
    steps = getattr(schedules, schedule)(reqs, tail=5) if schedule != "portions" else schedules.portions(reqs)
    got = _replay_cpu(folder, name, steps)
    expected = {rid: plain.forward(cfg, w, toks).numpy() for rid, toks in reqs.items()}
    assert sum(len(v) for v in got.values()) == sum(len(t) for t in reqs.values())
    bad = schedules.first_bad(got, expected, 2e-4)
    assert bad is None, f"first wrong place (request, position, error): {bad}"


def _changed(cfg, change):
    c = json.loads(json.dumps(cfg))
    change(c["layers"])
    return c


def test_the_tiny_models_show_a_mistake(tmp_path):
    """Each of these mistakes, planted in the plain model's configuration or weights, moves some logit of a tiny model by
    far more than the tolerances of the tests that compare the engine with the plain model."""
    def largest(name, n, cfg2=None, w2=None):
        folder = st.make_tiny_folder(name, tmp_path)
        cfg, w = plain.read_folder(folder)
        ids = st.random_ids(n, cfg["vocab"], 9)
        a = plain.forward(cfg, w, ids)
        b = plain.forward(cfg2(cfg) if cfg2 else cfg, w2(dict(w)) if w2 else w, ids)
        return float(((a - b).abs() / a.abs().amax()).max())

    mixer = lambda i, **kw: (lambda cfg: _changed(cfg, lambda l: l[i]["mixer"].update(kw)))
    mask = lambda i, **kw: (lambda cfg: _changed(cfg, lambda l: l[i]["mixer"]["mask"].update(kw)))
    mlp = lambda i, part, v: (lambda cfg: _changed(cfg, lambda l: l[i]["mlp"][part].update(limit=v)))
    cases = {
        "window one wider": ("A", 40, mask(0, size=8)), "window one narrower": ("A", 40, mask(2, size=20)),
        "one more kept": ("A", 40, mask(0, keep_first=4)), "one fewer kept": ("A", 60, mask(2, keep_first=17)),
        "none kept": ("C", 120, mask(0, keep_first=0)), "self and kept only": ("D", 40, mask(0, size=2)),
        "no cap": ("A", 20, mixer(0, softcap=None)), "plain frequencies": ("A", 40, lambda c: _changed(c, lambda l: l[0]["mixer"]["rot"].pop("scaling"))),
        "expert limit": ("A", 20, mlp(0, "expert", 0.9)), "shared limit": ("A", 20, mlp(1, "shared", 1.3)),
    }
    for what, (name, n, change) in cases.items():
        assert largest(name, n, change) > 5e-3, what

    def zero(key):
        def f(w):
            w[key] = torch.zeros_like(w[key])
            return w
        return f
    def other(key, fn):
        def f(w):
            w[key] = fn(w[key])
            return w
        return f
    weights = {
        "no head gate": ("A", 20, zero("l0.mix.g")), "recurrence gate": ("A", 20, zero("l1.mix.ra")), "input gate": ("A", 20, zero("l1.mix.ri")),
        "parts swapped": ("A", 20, other("l1.mix.ra", lambda t: t.flip(0))), "gate transposed": ("A", 20, other("l1.mix.ri", lambda t: t.transpose(1, 2))),
        "filter reversed": ("A", 20, other("l1.mix.conv", lambda t: t.flip(1))), "decays": ("A", 30, other("l1.mix.lam", lambda t: t + 0.2)),
        "table columns": ("A", 20, other("l0.mlp.table", lambda t: (t + 1) % 5)), "q norm": ("A", 20, other("l0.mix.q.norm", lambda t: torch.ones_like(t))),
        "norm weights": ("A", 20, zero("l1.norm1")), "gate bias": ("A", 20, zero("l1.mix.ra.b")), "filter bias": ("A", 20, zero("l1.mix.conv.b")),
    }
    for what, (name, n, change) in weights.items():
        assert largest(name, n, None, change) > 5e-3, what


def test_the_plain_functions_agree_with_closed_forms():
    f64 = torch.float64
    # an output norm: unit rows times 1 + w
    x = torch.tensor([[3.0, -3.0, 3.0, -3.0]], dtype=f64)
    assert torch.allclose(plain.zero_centred_norm(x, torch.full((4,), 0.5, dtype=f64), 0.0), torch.tensor([[1.5, -1.5, 1.5, -1.5]], dtype=f64))
    assert torch.allclose(plain.zero_centred_norm(x, torch.zeros(4, dtype=f64), 16.0), x / 5.0)
    # visible keys: itself, the window, the first ones; never the future
    ok = plain.visible(9, {"size": 3, "keep_first": 2})
    assert ok[8].tolist() == [True, True, False, False, False, False, True, True, True]
    assert ok[3].tolist() == [True, True, True, True] + [False] * 5 and ok[0].tolist() == [True] + [False] * 8
    assert plain.visible(4, None).sum() == 10
    # a rotation by p and back is the identity; half a turn swaps signs
    v = torch.randn(5, 2, 6, dtype=f64)
    pos = torch.tensor([0, 1, 7, 100, 5000])
    fr = plain.plain_frequencies(50.0, 6)
    assert torch.allclose(plain.rotate_halves(plain.rotate_halves(v, pos, fr), pos, fr, sign=-1.0), v, atol=1e-9)
    assert torch.allclose(plain.rotate_halves(v[:1], torch.tensor([1]), [math.pi] * 3), -v[:1], atol=1e-12)
    # turned values: one key alone comes back turned by the distance only
    for j, i in ((0, 3), (10, 13), (1000, 1003)):
        there = plain.rotate_halves(v[:1], torch.tensor([j]), fr)
        back = plain.rotate_halves(there, torch.tensor([i]), fr, sign=-1.0)
        assert torch.allclose(back, plain.rotate_halves(v[:1], torch.tensor([3]), fr, sign=-1.0), atol=1e-9)
    # the blend: often-turning pairs keep their frequency, seldom-turning ones are slowed, the magnitude is 1 + 0.1 ln(factor)
    f, mag = plain.key_frequencies(10000.0, 32, {"factor": 4.0, "original": 1024.0, "fast": 32.0, "slow": 1.0})
    p0 = plain.plain_frequencies(10000.0, 32)
    assert f[0] == p0[0] and abs(f[-1] - p0[-1] / 4.0) < 1e-15 and abs(mag - (1 + 0.1 * math.log(4.0))) < 1e-12
    assert any(p / 4.0 < a < p for a, p in zip(f, p0))
    # equal keys: the mean of the visible values
    q, k = torch.ones(4, 1, 2, dtype=f64), torch.ones(4, 1, 2, dtype=f64)
    vals = torch.tensor([1.0, 10.0, 100.0, 1000.0], dtype=f64).view(4, 1, 1)
    got = plain.softmax_attention(q, k, vals, 0.5, 2.0, {"size": 2, "keep_first": 1})[:, 0, 0]
    assert torch.allclose(got, torch.tensor([1.0, 5.5, 37.0, (1 + 100 + 1000) / 3], dtype=f64))
    # the recurrence: r = 1, i = 1, constant input u: S_t = u sqrt(1 - a^2) (1 - a^t) / (1 - a)
    lam = torch.tensor([-3.0], dtype=f64)
    a = math.exp(-8.0 * math.log1p(math.exp(-3.0)))
    one = torch.ones(6, 1, dtype=f64)
    S = plain.gated_recurrence(2.0 * one, one, one, lam)[:, 0]
    want = [2.0 * math.sqrt(1 - a * a) * (1 - a ** t) / (1 - a) for t in range(1, 7)]
    assert torch.allclose(S, torch.tensor(want, dtype=f64))
    # block gates: every part sees its own channels only
    u = torch.randn(3, 6, dtype=f64)
    w = torch.randn(3, 2, 2, dtype=f64)
    full = torch.block_diag(*w)
    assert torch.allclose(plain.block_gate(u, w, torch.zeros(3, 2, dtype=f64)), torch.sigmoid(u @ full.T))
    # the clamped unit: gate far above and up far below the limit
    W = {"gate": torch.tensor([[50.0]], dtype=f64), "up": torch.tensor([[-50.0]], dtype=f64), "down": torch.tensor([[1.0]], dtype=f64)}
    got = float(plain.clamped_expert(torch.ones(1, 1, dtype=f64), W, "", 2.0))
    assert abs(got - 2.0 / (1 + math.exp(-3.404)) * (1 - 2.0)) < 1e-12
    # equal experts by table: the mean; the shared one is added whole
    E = {f"e{e}.{n}": torch.full((1, 1), s, dtype=f64) for e, s in enumerate((1.0, 2.0, 3.0)) for n in ("gate", "up", "down")}
    E["table"] = torch.tensor([[0, 2], [1, 0]], dtype=torch.int32)
    ff = {"router": {"experts": 3, "top": 2}, "expert": {"limit": 9.0}}
    x = torch.ones(3, 1, dtype=f64)
    one_of = lambda e: plain.clamped_expert(x[:1], E, f"e{e}.", 9.0)[0]
    got = plain.table_moe(x, torch.tensor([1, 0, 1]), E, "", ff)
    assert torch.allclose(got, torch.stack([(one_of(1) + one_of(0)) / 2, (one_of(0) + one_of(2)) / 2, (one_of(1) + one_of(0)) / 2]))
    E.update({f"shared.{n}": torch.full((1, 1), 0.5, dtype=f64) for n in ("gate", "up", "down")})
    ff["shared"] = {"limit": 0.1}
    assert torch.allclose(plain.table_moe(x, torch.tensor([1, 0, 1]), E, "", ff) - got, plain.clamped_expert(x, E, "shared.", 0.1))
