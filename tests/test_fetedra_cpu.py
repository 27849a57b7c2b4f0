"""Fetedra without a GPU: the parser and its refusals, checkpoint names, a size that only the tensors give, the memory the two
mixers declare, the engine's host logic (portions down to two tokens, mixed batches, pages and slots used again) through the
kernel twins against the plain model, and the plain model's mechanisms against closed forms."""

from __future__ import annotations

import json
import math

import pytest
import torch
from safetensors.torch import load_file, save_file

from tests import fetedra_tiny as ft
from tests import plain_fetedra as plain
from tests import schedules
from turingserve_b200.config.model_config import (
    GatedMLPSpec, HalfRotarySpec, LatentAttentionSpec, RoutedMLPSpec, StreamLinkSpec, WKVSpec)
from turingserve_b200.config.registry import get_architecture, load_model_config
from turingserve_b200.parts.base import BuildContext, CacheNeed, ParamSpec, StateNeed, build


def test_parser_reads_every_size_and_option():
    cfg = ft.tiny_config("A")
    assert cfg.architecture == "Fetedra" and (cfg.hidden_size, cfg.vocab_size) == (60, 131) and cfg.tie_word_embeddings
    assert [r.layer for r in cfg.schedule] == [0, 1, 2, 3] and cfg.final_norm.eps == 1e-5 and cfg.final_norm.weight_offset == 1.0
    assert cfg.final_norm.streams == 3 and cfg.extra("logit_scale") == 0.7 and cfg.extra("streams") == 3
    assert cfg.layers[0].mixer == LatentAttentionSpec(
        num_heads=3, nope_dim=10, rope_dim=6, value_dim=12, q_rank=20, kv_rank=28, scale=0.4, norm_eps=1e-5,
        position=HalfRotarySpec(base=100.0, dims=6), window=7, sinks=True, head_gate=True)
    assert cfg.layers[0].mixer_link == StreamLinkSpec(streams=3, learned=True)
    assert cfg.layers[1].mixer == WKVSpec(num_heads=3, head_dim=20, norm_eps=1e-5, decay_rank=12)
    assert cfg.layers[2].mixer.position == HalfRotarySpec(base=40.0, dims=6) and cfg.layers[2].mixer.rope_dim == 10
    f = cfg.layers[0].feed_forward
    assert isinstance(f, RoutedMLPSpec) and (f.num_experts, f.top_k, f.intermediate_size, f.shared_intermediate_size) == (12, 3, 20, 28)
    assert (f.groups, f.groups_kept, f.weight_scale, f.correction, f.shared_gate, f.renormalize) == (4, 2, 1.7, True, True, True)
    assert (f.glu_limit, f.shared_glu_limit, f.glu_slope, f.glu_offset, f.scoring, f.weight_on) == (0.6, 0.9, 1.702, 1.0, "sigmoid", "output")
    d = cfg.layers[1].feed_forward
    assert isinstance(d, GatedMLPSpec) and d.intermediate_size == 52 and d.activation == "silu"
    assert "feed_forward" not in cfg.layers[2].roles
    g = cfg.layers[3].feed_forward
    assert g.shared_intermediate_size is None and not g.shared_gate
    plain_sum = ft.tiny_config("D")
    assert plain_sum.layers[0].mixer_link == StreamLinkSpec(streams=1, learned=False) and plain_sum.extra("streams") is None
    assert ft.tiny_config("B").layers[3].mixer.window is None


def test_names_round_trip_and_registry(tmp_path):
    arch = get_architecture("Fetedra")
    for name in ft.TINY:
        cfg = ft.tiny_config(name)
        assert arch.parse_config(json.loads(json.dumps(arch.to_config_json(cfg)))) == cfg
        loaded = load_model_config(ft.make_tiny_folder(name, tmp_path))
        assert [l.roles.keys() for l in loaded.layers] == [l.roles.keys() for l in cfg.layers]
    cfg = ft.tiny_config("A")
    names = set(arch.build_model(cfg, torch.float32, "cpu", 1).parameters(arch.tensor_names(cfg)))
    assert {"embed", "final.norm", "l0.norm1", "l0.norm2", "l0.hc1.in", "l0.hc1.out", "l0.hc1.mix", "l0.hc2.in", "l0.mix.dq",
            "l0.mix.dq.norm", "l0.mix.uq", "l0.mix.dkv", "l0.mix.dkv.norm", "l0.mix.uk", "l0.mix.uv", "l0.mix.sink", "l0.mix.g",
            "l0.mix.o", "l0.mlp.router", "l0.mlp.correction", "l0.mlp.e11.gate", "l0.mlp.e11.up", "l0.mlp.e11.down",
            "l0.mlp.shared.gate", "l0.mlp.shared.up", "l0.mlp.shared.down", "l0.mlp.shared.sg", "l1.mix.mu.r", "l1.mix.mu.k",
            "l1.mix.mu.v", "l1.mix.mu.g", "l1.mix.mu.w", "l1.mix.r", "l1.mix.k", "l1.mix.v", "l1.mix.g", "l1.mix.w1", "l1.mix.w2",
            "l1.mix.w0", "l1.mix.u", "l1.mix.norm", "l1.mix.o", "l1.mlp.gate", "l1.mlp.up", "l1.mlp.down"} <= names
    assert not {"l2.norm2", "l2.hc2.in", "l3.mlp.shared.up", "l3.mlp.shared.sg", "head"} & names
    d = ft.tiny_config("D")
    assert not any(".hc" in n for n in arch.build_model(d, torch.float32, "cpu", 1).parameters(arch.tensor_names(d)))


def test_parser_refusals():
    ok = ft.TINY["D"][0]

    def refused(change, text):
        layers = json.loads(json.dumps(ok["layers"]))
        change(layers)
        with pytest.raises(ValueError, match=text):
            get_architecture("Fetedra").build_model(ft.make_config(**{**ok, "layers": layers}), torch.float32, "cpu", 1)

    refused(lambda l: l[0].update(type="conv"), "unknown layer type")
    refused(lambda l: l[0]["mlp"].update(kind="sparse"), "unknown feed-forward")
    refused(lambda l: l[0]["mixer"].pop("scale"), "scale")
    refused(lambda l: l[0]["mixer"]["mask"].pop("size"), "size")
    refused(lambda l: l[0]["mixer"]["rot"].update(dims=8), "rot.dims")
    refused(lambda l: l[0]["mixer"].update(kv_rank=640), "cached rows")
    refused(lambda l: l[1]["mixer"].update(dim=300), "heads of up to")
    refused(lambda l: l[0]["mlp"]["router"].update(top=3), "top 3 of 2")
    refused(lambda l: l[0]["mlp"]["router"].update(groups={"count": 2, "keep": 3}), "groups")
    refused(lambda l: l[0]["mlp"]["router"].update(groups={"count": 2, "keep": 1}), "top 2 of 1 groups")
    refused(lambda l: l[0]["mlp"]["expert"].pop("limit"), "limit")
    with pytest.raises(ValueError, match="streams"):
        ft.make_config(**{**ok, "streams": 0})


def test_the_rank_of_the_decay_is_the_tensors(tmp_path):
    """No key names it: the same configuration loads with another rank, and two tensors that disagree are refused."""
    from turingserve_b200.weights.loader import WeightsError, load_model
    folder = ft.make_tiny_folder("D", tmp_path)
    assert load_model_config(folder).layers[1].mixer.decay_rank is None
    model, _ = load_model(folder, torch.float32, "cpu", 8)
    assert tuple(model.blocks[1].mixer.w1.shape) == (9, 32) and tuple(model.blocks[1].mixer.w2.shape) == (24, 9)
    path = f"{folder}/model.safetensors"
    t = load_file(path)
    t["l1.mix.w1"], t["l1.mix.w2"] = torch.ones(4, 32), torch.ones(24, 4)
    save_file(t, path)
    model, _ = load_model(folder, torch.float32, "cpu", 8)
    assert tuple(model.blocks[1].mixer.w1.shape) == (4, 32)
    t["l1.mix.w2"] = torch.ones(24, 5)
    save_file(t, path)
    with pytest.raises(ValueError, match="w1 has 4 rows"):
        load_model(folder, torch.float32, "cpu", 8)
    t["l1.mix.w1"] = torch.ones(4, 33)
    save_file(t, path)
    with pytest.raises(WeightsError, match="wrong shapes"):
        load_model(folder, torch.float32, "cpu", 8)
    spec = ParamSpec((None, 6), free=3)
    assert spec.fits((7, 6)) and not spec.fits((7, 5)) and not spec.fits((7,)) and spec.sizes == (3, 6)


def test_memory_of_every_run():
    from turingserve_b200.engine.runner import run_needs
    model = get_architecture("Fetedra").build_model(ft.tiny_config("A"), torch.float32, "cpu", 1)
    needs = run_needs(model)
    assert needs[0].cache == CacheNeed(1, 34, 7, value_dim=0) and needs[0].state is None
    assert needs[1].cache is None and needs[1].state == StateNeed((3 * 20 * 20 + 60,), torch.float32)
    assert needs[2].cache == CacheNeed(1, 28, 21, value_dim=0)
    assert needs[3].state == StateNeed((-(-(2 * 7 * 7 + 60) // 4) * 4,), torch.float32)


def test_parts_refuse_what_they_have_no_kernel_for():
    ctx = BuildContext(16, torch.float32, torch.device("cpu"), 0)
    base = dict(num_experts=4, top_k=2, intermediate_size=8, activation="clamped_glu", gated=True, weight_on="output")
    with pytest.raises(ValueError, match="shared expert's gate"):
        build("feed_forward", RoutedMLPSpec(**base, shared_gate=True), ctx)
    with pytest.raises(ValueError, match="groups"):
        build("feed_forward", RoutedMLPSpec(**base, groups=3, groups_kept=1), ctx)
    with pytest.raises(ValueError, match="table of experts"):
        build("feed_forward", RoutedMLPSpec(**base, table_rows=5, weight_scale=2.0), ctx)


def _replay_cpu(folder, name, steps, page=None):
    from turingserve_b200 import kernels
    from turingserve_b200.engine.replay import Replayer
    from tests.twin_ops import TwinOps
    kernels.use(TwinOps())
    try:
        rp = Replayer(folder, torch.float32, schedules.peak_tokens(steps), "cpu", page_size=page or ft.page_size(name))
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
    portions down to two tokens that end in the middle of pages and windows."""
    folder = ft.make_tiny_folder(name, tmp_path)
    cfg, w = plain.read_folder(folder)
    reqs = {f"r{i}": ft.random_ids(n, cfg["vocab"], 50 + i) for i, n in enumerate([1, 9, 34, 21, 17, 46])}
    steps = getattr(schedules, schedule)(reqs, tail=5) if schedule != "portions" else schedules.portions(reqs)
    got = _replay_cpu(folder, name, steps)
    expected = {rid: plain.forward(cfg, w, toks).numpy() for rid, toks in reqs.items()}
    assert sum(len(v) for v in got.values()) == sum(len(t) for t in reqs.values())
    bad = schedules.first_bad(got, expected, 3e-4)
    assert bad is None, f"first wrong place (request, position, error): {bad}"


def test_the_tiny_models_show_a_mistake(tmp_path):
    """Each of these mistakes, planted in the plain model's configuration or weights, moves some logit of a tiny model by
    far more than the tolerances of the tests that compare the engine with the plain model."""
    def largest(name, n, change, w_change=None):
        folder = ft.make_tiny_folder(name, tmp_path)
        cfg, w = plain.read_folder(folder)
        ids = ft.random_ids(n, cfg["vocab"], 9)
        a = plain.forward(cfg, w, ids)
        c = json.loads(json.dumps(cfg))
        if change:
            change(c)
        w2 = dict(w)
        if w_change:
            w_change(w2)
        return float(((a - plain.forward(c, w2, ids)).abs() / a.abs().amax()).max())

    mixer = lambda i, **kw: (lambda c: c["layers"][i]["mixer"].update(kw))
    router = lambda i, **kw: (lambda c: c["layers"][i]["mlp"]["router"].update(kw))
    cases = {
        "window one wider": ("A", 40, mixer(0, mask={"size": 8})), "window one narrower": ("A", 40, mixer(2, mask={"size": 20})),
        "no window": ("B", 60, mixer(2, mask=None)), "itself and the one before": ("D", 12, mixer(0, mask={"size": 2})),
        "scale": ("A", 20, mixer(0, scale=0.5)), "rotation base": ("A", 40, mixer(0, rot={"base": 120.0, "dims": 6})),
        "whole rotated part turned": ("A", 40, mixer(2, rot={"base": 40.0, "dims": 10})),
        "expert limit": ("A", 20, lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.7)),
        "shared limit": ("A", 20, lambda c: c["layers"][0]["mlp"]["shared"].update(limit=1.0)),
        "other groups": ("A", 20, router(0, groups={"count": 4, "keep": 3})), "no groups": ("A", 20, router(0, groups={"count": 1, "keep": 1})),
        "weight scale": ("A", 20, router(0, scale=1.6)), "logit scale": ("A", 5, lambda c: c.update(logit_scale=0.71)),
    }
    for what, (name, n, change) in cases.items():
        assert largest(name, n, change) > 5e-3, what
    scaled = lambda key, f: (lambda w: w.update({key: f(w[key])}))
    zero = lambda t: torch.zeros_like(t)
    weights = {
        "no head gate": ("A", 20, "l0.mix.g", zero), "no sink": ("A", 20, "l0.mix.sink", lambda t: t - 50.0),
        "sinks moved on": ("A", 20, "l0.mix.sink", lambda t: t.roll(1)), "no correction": ("A", 20, "l0.mlp.correction", zero),
        "shared gate": ("A", 20, "l0.mlp.shared.sg", zero), "mix transposed": ("A", 20, "l0.hc1.mix", lambda t: t.T),
        "out weights": ("A", 20, "l1.hc2.out", lambda t: t.flip(0)), "no shift of r": ("A", 20, "l1.mix.mu.r", zero),
        "no shift of the decay": ("A", 20, "l1.mix.mu.w", zero), "no shift of the gate": ("A", 20, "l1.mix.mu.g", zero),
        "no bonus": ("A", 20, "l1.mix.u", zero), "bonus of another head": ("A", 20, "l1.mix.u", lambda t: t.roll(1, 0)),
        "plain decay": ("A", 20, "l1.mix.w2", zero), "decay base": ("A", 30, "l1.mix.w0", lambda t: t + 0.2),
        "heads' norm": ("A", 20, "l1.mix.norm", torch.ones_like), "query latent's norm": ("A", 20, "l0.mix.dq.norm", torch.ones_like),
        "key latent's norm": ("A", 20, "l0.mix.dkv.norm", torch.ones_like), "norm weights": ("A", 20, "l1.norm1", zero),
        "a forgotten state": ("B", 60, "l1.mix.w0", lambda t: t + 4.0),
    }
    for what, (name, n, key, f) in weights.items():
        assert largest(name, n, None, scaled(key, f)) > 5e-3, what


def test_the_plain_functions_agree_with_closed_forms():
    f64 = torch.float64
    x = torch.tensor([[3.0, -3.0, 3.0, -3.0]], dtype=f64)
    assert torch.allclose(plain.zero_centred_norm(x, torch.full((4,), 0.5, dtype=f64), 0.0), torch.tensor([[1.5, -1.5, 1.5, -1.5]], dtype=f64))
    assert torch.allclose(plain.unit_rms(x, 16.0), x / 5.0)
    # mixes: mu 0 is the row itself, mu 1 the row before, zeros before the first
    h = torch.randn(4, 3, dtype=f64)
    assert torch.equal(plain.shifted_mix(h, torch.zeros(3, dtype=f64)), h)
    one = plain.shifted_mix(h, torch.ones(3, dtype=f64))
    assert torch.allclose(one[1:], h[:-1]) and torch.allclose(one[0], torch.zeros(3, dtype=f64))
    # a decay from w0 alone
    d = plain.decay_of(torch.randn(2, 3, dtype=f64), torch.zeros(2, 3, dtype=f64), torch.randn(4, 2, dtype=f64), torch.full((4,), math.log(0.25), dtype=f64))
    assert torch.allclose(d, torch.full((2, 4), math.exp(-0.25), dtype=f64))
    # one channel, constant k, v, r = 1 and decay a: o_t = u + (1 - a^t) / (1 - a), S_T = (1 - a^T) / (1 - a)
    ones = torch.ones(6, 1, 1, dtype=f64)
    a, u = 0.7, 0.3
    o, S = plain.fading_state_scan(ones, ones, ones, a * ones, torch.full((1, 1), u, dtype=f64))
    assert torch.allclose(o[:, 0, 0], torch.tensor([u + (1 - a ** t) / (1 - a) for t in range(6)], dtype=f64))
    assert torch.allclose(S[0, 0, 0], torch.tensor((1 - a ** 6) / (1 - a), dtype=f64))
    # ... and carried on from a state the sequence is the same
    r, k, w = (torch.rand(7, 2, 3, dtype=f64) for _ in range(3))
    v, bonus = torch.randn(7, 2, 5, dtype=f64), torch.randn(2, 3, dtype=f64)
    whole, last = plain.fading_state_scan(r, k, v, w, bonus)
    head, mid = plain.fading_state_scan(r[:3], k[:3], v[:3], w[:3], bonus)
    tail, end = plain.fading_state_scan(r[3:], k[3:], v[3:], w[3:], bonus, mid)
    assert torch.allclose(torch.cat([head, tail]), whole) and torch.allclose(end, last)
    # a rotation there and back; half a turn; pairs are (i, i + dims / 2), the rest passes
    z = torch.randn(3, 2, 8, dtype=f64)
    pos = torch.tensor([0, 3, 5000])
    turned = plain.rotate_halves(z, pos, 50.0, 6)
    assert torch.allclose(turned[0], z[0]) and torch.equal(turned[..., 6:], z[..., 6:])
    assert torch.allclose(plain.rotate_halves(turned, -pos, 50.0, 6), z, atol=1e-9)
    assert torch.allclose(turned[1, 0, 0], z[1, 0, 0] * math.cos(3) - z[1, 0, 3] * math.sin(3))
    assert plain.visible(5, 2).tolist()[3] == [False, False, True, True, False] and plain.visible(4, None).sum() == 10
    # equal scores of zero and a sink of ln 2: n keys weigh 1 / (n + 2) each
    p = plain.sink_softmax(torch.zeros(3, 3, dtype=f64), plain.visible(3, None), torch.tensor(math.log(2.0), dtype=f64))
    assert torch.allclose(p[2], torch.full((3,), 0.2, dtype=f64)) and torch.allclose(p[0], torch.tensor([1 / 3, 0.0, 0.0], dtype=f64))
    # groups: the single best expert lies in a group whose sum of two is smaller; corrections make scores negative
    s = torch.tensor([0.9, 0.1, 0.6, 0.55, 0.2, 0.3])
    c = torch.tensor([-1.0] * 6)
    assert plain.choose(s, c, 2, 3, 1) == [2, 3] and plain.choose(s, c, 2, 1, 1) == [0, 2] and plain.choose(s, c, 3, 3, 2) == [0, 2, 3]
    assert plain.choose(s, torch.tensor([0.0, 0, 0, 0, 0.9, 0.9]), 2, 6, 3) == [5, 4]
    # streams: mix [from, to], all copies from the old ones
    xs = [torch.tensor([1.0, 2.0]), torch.tensor([10.0, 20.0])]
    new = plain.write_streams(xs, torch.tensor([100.0, 0.0]), torch.tensor([[1.0, 0.5], [0.0, 2.0]]), torch.tensor([1.0, -1.0]))
    assert new[0].tolist() == [101.0, 2.0] and new[1].tolist() == [0.5 + 20.0 - 100.0, 1.0 + 40.0]
    assert plain.read_streams(xs, torch.tensor([2.0, -1.0])).tolist() == [-8.0, -16.0]
    W = {"gate": torch.tensor([[50.0]], dtype=f64), "up": torch.tensor([[-50.0]], dtype=f64), "down": torch.tensor([[1.0]], dtype=f64)}
    got = float(plain.clamped_expert(torch.ones(1, 1, dtype=f64), W, "", 2.0))
    assert abs(got - 2.0 / (1 + math.exp(-3.404)) * (1 - 2.0)) < 1e-12
