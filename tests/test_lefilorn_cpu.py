"""Lefilorn without a GPU: the configuration reader and its plan, the tensors the model names, what the cache keeps, and the plain
implementation's mechanisms on cases worked out by hand."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_lefilorn as plain
from lefilorn_models import CONFIGS, make_weights, tensor_shapes


def test_configuration_round_trip_and_plan():
    from pico_engine.config import (BranchSumSpec, ConfigError, GatedAttentionSpec, GatedMLPSpec, LinearAttentionSpec, RMSNormSpec,
                                    RotaryHalvesSpec, RotaryPairsSpec, StreamMixSpec, config_from_dict)
    for name, d in CONFIGS.items():
        cfg = config_from_dict(copy.deepcopy(d))
        assert config_from_dict(cfg.to_dict()) == cfg and {k: v for k, v in cfg.to_dict().items() if k != "layers"} == {k: v for k, v in d.items() if k != "layers"}
        plan = cfg.plan()
        assert plan.embedding_scale == d["embedding"]["scale"] and plan.head == "head" and type(plan.final_norm) is RMSNormSpec
        assert plan.streams == d.get("streams") and [e.layer for e in plan.schedule] == plain.layer_runs(d)
        assert all(e.cache_of is None and not e.add_embedding and e.add_vector is None for e in plan.schedule)
        for i, (l, spec) in enumerate(zip(d["layers"], plan.layers)):
            a, b = l["mixer"]["left"], l["mixer"]["right"]
            assert type(spec.mixer) is BranchSumSpec and spec.mixer.out_norms is None
            assert spec.mixer.scales == (l["mixer"]["left_scale"], l["mixer"]["right_scale"])
            att, ret = spec.mixer.branches
            assert type(att) is GatedAttentionSpec and type(att.position) is RotaryPairsSpec and att.position.dims == a["rot"]["dims"]
            assert (att.window, att.keep_first) == ((a.get("mask") or {}).get("size"), (a.get("mask") or {}).get("keep_first", 0))
            assert att.bias and not att.o_bias and att.qk_row_norm == ("q.norm", "k.norm") and att.gate == "g"
            assert type(ret) is LinearAttentionSpec and type(ret.position) is RotaryHalvesSpec and ret.position.dims == b["rot"]["dims"]
            assert ret.head_decay == tuple(b["decay"]) and ret.k_scale == b["dim"] ** -0.5 and ret.norm_name is None and ret.norm_over == "head"
            assert spec.arrangement == ("pre_norm" if "streams" not in d else "streams")
            if "streams" in d:
                assert spec.mixer_streams == StreamMixSpec(d["streams"], f"l{i}.hc1.in", f"l{i}.hc1.out", f"l{i}.hc1.mix")
            assert (spec.feed_forward is None) == (l["mlp"] is None)
            assert (spec.feed_forward_streams is None) == (l["mlp"] is None or "streams" not in d)
            if l["mlp"] is not None:
                assert type(spec.feed_forward) is GatedMLPSpec and spec.feed_forward.activation == "relu"

    def broken(name, change, match):
        bad = copy.deepcopy(CONFIGS[name])
        change(bad)
        with pytest.raises(ConfigError, match=match):
            config_from_dict(bad).plan()
    broken("L1", lambda c: c["layers"][1].update(type="mamba"), "type")
    broken("L1", lambda c: c["layers"][0]["mixer"].pop("right"), "right")
    broken("L1", lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale")
    broken("L1", lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=34), "rot.dims")
    broken("L1", lambda c: c["layers"][0]["mixer"]["right"]["rot"].update(dims=7), "rot.dims")
    broken("L1", lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "evenly")
    broken("L1", lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]), "decay")
    broken("L1", lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask.size")
    broken("L1", lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first")
    broken("L1", lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind")
    broken("L1", lambda c: c["loop"].update(stop=4), "loop")
    broken("L1", lambda c: c["loop"].update(times=0), "loop")
    broken("L1", lambda c: c.update(streams=0), "streams")
    broken("L1", lambda c: c.pop("width"), "width")


def test_the_model_names_the_tensors_of_the_design():
    from pico_engine.config import ConfigError, config_from_dict
    from pico_engine.config.registry import architecture
    from pico_engine.weights.loader import WeightError, check
    for name, d in CONFIGS.items():
        model = architecture("Lefilorn").build_model(config_from_dict(d), torch.bfloat16, "meta")
        stored = tensor_shapes(d)
        assert {k: tuple(v.shape) for k, v in model.expected_tensors().items()} == stored, name
        check(model.expected_tensors(), stored, model.plan.ignorable_tensors)
        lacking = dict(stored); lacking.pop("l0.mix.left.q.norm")
        with pytest.raises(WeightError, match="l0.mix.left.q.norm"):
            check(model.expected_tensors(), lacking, model.plan.ignorable_tensors)
        needs = model.cache_needs()
        assert len(needs) == len(plain.layer_runs(d))
        for i, need in zip(plain.layer_runs(d), needs):
            a, b = d["layers"][i]["mixer"]["left"], d["layers"][i]["mixer"]["right"]
            mask = a.get("mask") or {}
            assert (need.kv.n_kv_heads, need.kv.head_dim, need.kv.value_shape) == (a["kv_heads"], a["dim"], (a["kv_heads"], a["vdim"]))
            assert (need.kv.window, need.kv.keep_first) == (mask.get("size"), mask.get("keep_first", 0))
            assert need.state_elems == b["heads"] * b["dim"] * b["vdim"] and need.state_dtype == "float32"
    # a layer without a feed-forward may store what would stand around it
    extra = dict(tensor_shapes(CONFIGS["L1"]), **{"l2.norm2": (72,), "l2.hc2.in": (2,), "l2.hc2.out": (2,), "l2.hc2.mix": (2, 2)})
    model = architecture("Lefilorn").build_model(config_from_dict(CONFIGS["L1"]), torch.bfloat16, "meta")
    check(model.expected_tensors(), extra, model.plan.ignorable_tensors)
    with pytest.raises(ConfigError, match="streams"):
        architecture("Lefilorn").build_model(config_from_dict(dict(CONFIGS["L1"], streams=33)), torch.bfloat16, "meta")


def test_parts_refuse_what_they_do_not_compute():
    from dataclasses import replace
    from pico_engine.config import ConfigError, LayerSpec, ModelPlan, RMSNormSpec, RotaryHalvesSpec, ScheduleEntry, config_from_dict
    from pico_engine.parts import BranchSum, GatedAttention, LinearAttention
    both = config_from_dict(CONFIGS["L1"]).plan().layers[0].mixer
    att, ret = both.branches
    f32 = (torch.float32, "meta")
    BranchSum(both, *f32)
    for spec, match in ((replace(att, qk_unit_norm=True), "norm"), (replace(att, position=RotaryHalvesSpec(32, 16, 100.0, (2.0, 8.0, 4.0, 1.0))), "stretched")):
        with pytest.raises(ConfigError, match=match):
            GatedAttention(spec, *f32)
    for spec, match in ((replace(ret, qk_activation="silu"), "activation"), (replace(ret, position=RotaryHalvesSpec(16, 18, 100.0)), "fit")):
        with pytest.raises(ConfigError, match=match):
            LinearAttention(spec, *f32)
    with pytest.raises(ConfigError, match="factor"):
        BranchSum(replace(both, scales=(1.0,)), *f32)
    plan = config_from_dict(CONFIGS["L1"]).plan()
    with pytest.raises(ConfigError, match="streams"):
        replace(plan, streams=3).validate()
    with pytest.raises(ConfigError, match="streams"):
        replace(plan, schedule=(ScheduleEntry(0, add_embedding=True),)).validate()
    with pytest.raises(ConfigError, match="streams"):
        ModelPlan("x", 8, 72, "e", (LayerSpec(both, RMSNormSpec(72, 1e-5, "n"), arrangement="streams"),), (ScheduleEntry(0),),
                  RMSNormSpec(72, 1e-5, "n"), None, 64).validate()


def test_first_pages_stay_and_the_others_leave_with_the_window():
    from pico_engine.cache import Cache
    from pico_engine.config import config_from_dict
    from pico_engine.config.registry import architecture
    model = architecture("Lefilorn").build_model(config_from_dict(CONFIGS["L3"]), torch.float32, "meta")
    cache = Cache(model.cache_needs(), 64 * 12, 2, torch.float32, "cpu", allocate=False)
    groups = {(g.need.window, g.need.keep_first): g for g in cache.groups}
    assert set(groups) == {(70, 100), (130, 64), (45, 0)}
    s = cache.open()
    cache.reserve(s, 500); cache.advance(s, 500)
    # the next query stands at 500: windows of 70, 130 and 45 begin at 431 (page 6), 371 (page 5) and 456 (page 7)
    assert [p >= 0 for p in groups[(70, 100)].table[s]] == [True, True] + [False] * 4 + [True] * 2
    assert [p >= 0 for p in groups[(130, 64)].table[s]] == [True] + [False] * 4 + [True] * 3
    assert [p >= 0 for p in groups[(45, 0)].table[s]] == [False] * 7 + [True]
    cache.check()
    cache.close(s)
    assert all(g.pages.free_count == g.pages.n for g in cache.groups)


def test_shapes_and_fewer_layers():
    from pico_engine.config import config_from_dict
    from pico_engine.config.shapes import shape, with_layers
    for name in ("lefilorn-tiny", "lefilorn-0.5b", "lefilorn-7b"):
        config_from_dict(shape(name)).plan()
    assert [e.layer for e in config_from_dict(shape("lefilorn-tiny")).plan().schedule] == [0, 1, 1, 2]
    assert [e.layer for e in config_from_dict(with_layers(shape("lefilorn-tiny"), 2)).plan().schedule] == [0, 1, 1]
    assert [e.layer for e in config_from_dict(with_layers(shape("lefilorn-tiny"), 1)).plan().schedule] == [0]


# ------------------------------------------------------------------ the plain implementation on cases worked out by hand

def test_plain_mask_by_hand():
    rows = plain.visible(6, 2, 1).tolist()
    assert rows[0] == [True] + [False] * 5 and rows[1] == [True, True] + [False] * 4
    assert rows[4] == [True, False, False, True, True, False] and rows[5] == [True, False, False, False, True, True]
    assert plain.visible(4, 1, 0).tolist() == torch.eye(4).bool().tolist()
    assert plain.visible(3).tolist() == torch.tril(torch.ones(3, 3)).bool().tolist()
    assert plain.visible(4, 1, 9).tolist() == torch.tril(torch.ones(4, 4)).bool().tolist()       # kept tokens are still causal


def test_plain_norm_and_rotations_by_hand():
    x = torch.tensor([[3.0, 4.0, 0.0, 0.0]], dtype=torch.float64)
    assert torch.allclose(plain.rms_norm(x, torch.tensor([1.0, 2.0, 1.0, 1.0]).double(), 0.0), torch.tensor([[1.2, 3.2, 0.0, 0.0]]).double())
    assert torch.allclose(plain.unit_rms(x, 0.25 * 11), x / 3.0)                                   # eps inside the root: sqrt(6.25 + 2.75)
    u = torch.tensor([[[1.0, 5.0, 0.0, 6.0, 7.0]]] * 2, dtype=torch.float64)
    c1, s1, c2, s2 = math.cos(1.0), math.sin(1.0), math.cos(0.1), math.sin(0.1)
    r = plain.rotate_neighbours(u, 4, 100.0)
    assert torch.equal(r[0], u[0])
    assert torch.allclose(r[1, 0], torch.tensor([c1 - 5 * s1, 5 * c1 + s1, -6 * s2, 6 * c2, 7.0]).double())
    r = plain.rotate_halves(u, 4, 100.0)
    assert torch.allclose(r[1, 0], torch.tensor([c1, 5 * c2 - 6 * s2, s1, 6 * c2 + 5 * s2, 7.0]).double())


def test_plain_retention_by_hand():
    q = torch.tensor([[[1.0, 0.0]], [[1.0, 2.0]], [[0.0, 1.0]]], dtype=torch.float64)
    k = torch.tensor([[[2.0, 0.0]], [[0.0, 1.0]], [[1.0, 1.0]]], dtype=torch.float64)
    v = torch.tensor([[[1.0]], [[3.0]], [[5.0]]], dtype=torch.float64)
    # S: (2, 0), (1, 3), (0.5 + 5, 1.5 + 5)
    assert plain.retention(q, k, v, [0.5]).flatten().tolist() == [2.0, 7.0, 6.5]
    assert plain.retention(q, k, v, [0.0]).flatten().tolist() == [2.0, 6.0, 5.0]                    # decay 0: the token alone


def test_plain_streams_by_hand():
    xs = [torch.tensor([[1.0]]), torch.tensor([[10.0]])]
    assert float(plain.streams_in(xs, torch.tensor([2.0, 0.5]))) == 7.0
    mix = torch.tensor([[1.0, 0.25], [0.0, 2.0]])                                                    # [from, to]
    new = plain.streams_out(xs, torch.tensor([[100.0]]), mix, torch.tensor([1.0, -1.0]))
    assert [float(x) for x in new] == [101.0, 0.25 + 20.0 - 100.0]


def test_plain_streams_of_one_with_unit_weights_are_the_plain_residual():
    cfg = CONFIGS["L2"]
    w = {n: t.double() for n, t in make_weights(cfg, 3).items()}
    ones = {n: (torch.ones_like(t) if ".hc" in n else t) for n, t in w.items()}
    bare = {n: t for n, t in w.items() if ".hc" not in n}
    toks = [3, 9, 27, 81, 5]
    with torch.no_grad():
        a, b = plain.logits(toks, ones, cfg), plain.logits(toks, bare, {k: v for k, v in cfg.items() if k != "streams"})
    assert torch.allclose(a, b, atol=1e-12)


def test_plain_relu_gate_by_hand():
    w = {"p.gate": torch.tensor([[1.0], [-1.0]]), "p.up": torch.tensor([[2.0], [2.0]]), "p.down": torch.tensor([[1.0, 10.0]])}
    assert float(plain.relu_gated(torch.tensor([[3.0]]), w, "p.")) == 18.0 and float(plain.relu_gated(torch.tensor([[-3.0]]), w, "p.")) == -180.0


def test_plain_prefix_does_not_depend_on_what_follows():
    cfg = CONFIGS["L1"]
    w = {n: t.double() for n, t in make_weights(cfg, 3).items()}
    toks = torch.randint(0, cfg["vocab"], (60,), generator=torch.Generator().manual_seed(1)).tolist()
    with torch.no_grad():
        a, b = plain.logits(toks, w, cfg), plain.logits(toks[:47], w, cfg)
    assert torch.allclose(a[:47], b, atol=1e-10)
