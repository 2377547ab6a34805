"""Razelorn without a GPU: the configuration reader and its plan, the tensors' names, what the cache keeps, and the plain implementation's
mechanisms on cases worked out by hand."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_razelorn as plain
from razelorn_models import CONFIGS, make_weights, owner, tensor_shapes


def build(d, dtype=torch.bfloat16):
    from pico_engine.config import config_from_dict
    from pico_engine.config.registry import architecture
    return architecture("Razelorn").build_model(config_from_dict(d), dtype, "meta")


def test_configuration_round_trip_and_plan():
    from pico_engine.config import (ConfigError, DenseMLPSpec, DifferentialAttentionSpec, LayerNormSpec, MixtureSpec, NoPositionSpec,
                                    RotaryHalvesSpec, config_from_dict)
    for name, d in CONFIGS.items():
        cfg = config_from_dict(copy.deepcopy(d))
        assert cfg.to_dict() == d, name
        plan = cfg.plan()
        owners = [i for i in range(len(d["layers"])) if owner(d, i) == i]
        assert len(plan.layers) == len(owners) and len(plan.schedule) == len(d["layers"])
        assert [owners[e.layer] for e in plan.schedule] == [owner(d, i) for i in range(len(d["layers"]))]
        assert all(e.cache_of is None for e in plan.schedule)
        assert plan.embedding_scale == d["embedding"]["scale"] and plan.head == "head" and type(plan.final_norm) is LayerNormSpec
        for i, spec in zip(owners, plan.layers):
            m, mlp = d["layers"][i]["mixer"], d["layers"][i]["mlp"]
            assert spec.arrangement == "parallel_one_norm" and spec.mixer_norm.bias == f"l{i}.norm1.b" and spec.feed_forward_norm is None
            a = spec.mixer
            assert type(a) is DifferentialAttentionSpec and (a.window, a.lambda_base, a.out_scale) == ((m.get("mask") or {}).get("size"), m["diff"], 1 - m["diff"])
            rot = m.get("rot")
            if rot is None or not rot["dims"]:
                assert type(a.position) is NoPositionSpec
            else:
                sc = rot.get("scaling")
                assert type(a.position) is RotaryHalvesSpec and a.position.stretch is None
                assert a.position.bands == (None if sc is None else (sc["factor"], sc["low"], sc["high"], sc["original"]))
            if mlp is None:
                assert spec.feed_forward is None
            elif mlp["kind"] == "dense":
                assert type(spec.feed_forward) is DenseMLPSpec and spec.feed_forward.activation == "relu2"
            else:
                f = spec.feed_forward
                assert type(f) is MixtureSpec and f.scores == "softmax_all" and f.correction_name == "correction"
                assert f.n_identity == mlp["router"].get("identity", 0) and f.shared_intermediate == (mlp.get("shared") or {}).get("ff")

    def broken(name, change, match):
        bad = copy.deepcopy(CONFIGS[name])
        change(bad)
        with pytest.raises(ConfigError, match=match):
            config_from_dict(bad)
    broken("R1", lambda c: c["layers"][1].update(type="mamba"), "type")
    broken("R1", lambda c: c["layers"][1]["mixer"].pop("diff"), "diff")
    broken("R1", lambda c: c["layers"][1]["mixer"]["rot"].update(dims=50), "rot.dims")
    broken("R1", lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(low=5.0), "low must lie below")
    broken("R1", lambda c: c["layers"][0]["mlp"]["router"].update(top=10), "exceeds")
    broken("R1", lambda c: c["layers"][3].update(weights_of=3), "weights_of")
    broken("R1", lambda c: c["layers"][3].update(weights_of=9), "weights_of")
    broken("R1", lambda c: c["layers"][0].update(weights_of=2), "weights_of")             # 0 and 2 would name each other
    broken("R1", lambda c: c["layers"][2].update(mlp=None), "is another")
    broken("R2", lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "evenly")
    broken("R2", lambda c: c["layers"][0]["mlp"].pop("expert"), "expert")


def test_parts_refuse_what_they_cannot_do():
    from pico_engine.config import (ConfigError, DifferentialAttentionSpec, LayerNormSpec, LayerSpec, MixtureSpec, NoPositionSpec, RotaryHalvesSpec)
    from pico_engine.parts import DifferentialAttention, Layer, Mixture
    from pico_engine.parts.attention_gated import halves_frequencies
    ok = dict(hidden=32, n_heads=2, n_kv_heads=1, head_dim=16, v_head_dim=16, window=None, scale=1.0, position=NoPositionSpec(), prefix="m.",
              lambda_base=0.1, out_scale=0.9)
    for change in (dict(n_heads=3, n_kv_heads=2), dict(head_dim=300), dict(window=0), dict(position=RotaryHalvesSpec(16, 18, 10.0)),
                   dict(position=RotaryHalvesSpec(16, 8, 10.0, stretch=(2.0, 8, 4.0, 1.0)))):
        with pytest.raises(ConfigError):
            DifferentialAttention(DifferentialAttentionSpec(**{**ok, **change}), torch.bfloat16, "meta")
    with pytest.raises(ConfigError, match="either"):
        halves_frequencies(RotaryHalvesSpec(16, 8, 10.0, stretch=(2.0, 8, 4.0, 1.0), bands=(2.0, 1.0, 4.0, 8)), "cpu")
    mix = dict(hidden=32, n_experts=4, top_k=2, intermediate=8, prefix="f.")
    for change in (dict(n_identity=1), dict(correction_name="c"), dict(scores="sigmoid", n_identity=1), dict(scores="softmax_all", n_groups=2),
                   dict(scores="softmax_all", n_identity=1, shared_intermediate=8, shared_gate_name=None)):
        with pytest.raises(ConfigError):
            Mixture(MixtureSpec(**{**mix, **change}), torch.bfloat16, "meta")
    norm = LayerNormSpec(32, 1e-5, "n", "n.b")
    with pytest.raises(ConfigError, match="one norm"):
        Layer(LayerSpec(DifferentialAttentionSpec(**ok), norm, MixtureSpec(**mix), norm, arrangement="parallel_one_norm"), torch.bfloat16, "meta")


def test_the_model_names_the_tensors_of_the_design():
    from pico_engine.weights.loader import check
    for name, d in CONFIGS.items():
        model = build(d)
        stored = tensor_shapes(d)
        assert {k: tuple(v.shape) for k, v in model.expected_tensors().items()} == stored, name
        check(model.expected_tensors(), stored, model.plan.ignorable_tensors)
        needs = model.cache_needs()
        assert len(needs) == len(d["layers"])                               # a layer on another's tensors has a cache of its own
        for l, need in zip(d["layers"], needs):
            m = l["mixer"]
            assert (need.kv.n_kv_heads, need.kv.head_dim, need.kv.value_shape, need.kv.window) == (2 * m["kv_heads"], m["dim"], (m["kv_heads"], m["vdim"]),
                                                                                                   (m.get("mask") or {}).get("size"))


def test_pages_leave_with_the_window():
    from pico_engine.cache import Cache
    cache = Cache(build(CONFIGS["R1"]).cache_needs(), 64 * 12, 2, torch.float32, "cpu", allocate=False)
    windows = {g.need.window: g for g in cache.groups}
    assert set(windows) == {70, 2} and windows[70].entries == [0, 2, 3]
    s = cache.open()
    cache.reserve(s, 500); cache.advance(s, 500)
    # the next query stands at 500: a window of 70 begins at 431 (page 6), one of 2 at 499 (page 7)
    assert [p >= 0 for p in windows[70].table[s]] == [False] * 6 + [True] * 2
    assert [p >= 0 for p in windows[2].table[s]] == [False] * 7 + [True]
    cache.check()
    cache.close(s)
    assert all(g.pages.free_count == g.pages.n for g in cache.groups)


def test_frequencies_of_the_part_equal_the_plain_ones():
    from pico_engine.config import RotaryHalvesSpec
    from pico_engine.parts.attention_gated import halves_frequencies
    for dims, base, sc in ((16, 1000.0, (4.0, 1.0, 4.0, 64)), (10, 100.0, (8.0, 0.5, 3.0, 40)), (48, 4e4, (8.0, 1.0, 2.0, 256)), (8, 50.0, None)):
        f, magnitude = halves_frequencies(RotaryHalvesSpec(dims, dims, base, bands=sc), "cpu")
        want = plain.frequencies(dims, base, None if sc is None else dict(zip(("factor", "low", "high", "original"), sc)))
        assert magnitude == 1.0 and torch.allclose(f.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6)


# ------------------------------------------------------------------ the plain implementation on cases worked out by hand

def t64(*rows):
    return torch.tensor(list(rows), dtype=torch.float64)


def test_plain_frequencies_by_hand():
    """base^(-1/2) steps of 1/10 from 1: wavelengths 6.28, 62.8, 628.  With original 300, low 1, high 10: below 30 kept, above 300 divided,
    62.8 in between with s = (300 / 62.8 - 1) / 9."""
    f = plain.frequencies(6, 1000.0, {"factor": 4.0, "low": 1.0, "high": 10.0, "original": 300})
    s = (300 / (20 * math.pi) - 1) / 9
    assert f[0] == 1.0 and abs(f[1] - ((1 - s) * 0.1 / 4 + s * 0.1)) < 1e-15 and abs(f[2] - 0.01 / 4) < 1e-15
    assert plain.frequencies(4, 100.0) == [1.0, 0.1]
    u = t64(*[[1.0, 5.0, 0.0, 6.0, 7.0]] * 2)
    r = plain.rotate_half(u, 4, [1.0, 0.1])
    assert torch.equal(r[0], u[0])
    c1, s1, c2, s2 = math.cos(1.0), math.sin(1.0), math.cos(0.1), math.sin(0.1)
    assert torch.allclose(r[1], t64(c1, 5 * c2 - 6 * s2, s1, 6 * c2 + 5 * s2, 7.0))


def test_plain_window_and_difference_by_hand():
    assert plain.window_mask(4, 2).tolist() == [[True, False, False, False], [True, True, False, False], [False, True, True, False], [False, False, True, True]]
    w = {"p.lq1": t64(1.0, 2.0), "p.lk1": t64(0.5, 0.0), "p.lq2": t64(0.0, 1.0), "p.lk2": t64(3.0, 0.25)}
    assert abs(float(plain.mixing_number(w, "p.", 0.3)) - (math.exp(0.5) - math.exp(0.25) + 0.3)) < 1e-12
    d = plain.difference_of_maps(t64([3.0, 5.0]), t64([0.0, 2.0]), 0.5, 0.2, 0.0)           # (3, 4) / sqrt(12.5) * 0.8
    assert torch.allclose(d, t64([3.0, 4.0]) / math.sqrt(12.5) * 0.8)
    # two keys; map 1 looks at the first, map 2 at the second: the output is v0 - lambda v1, normed
    q, k = torch.zeros(2, 1, 2, 1, dtype=torch.float64), torch.zeros(2, 1, 2, 1, dtype=torch.float64)
    q[1, 0, :, 0] = 100.0; k[0, 0, 0, 0] = 1.0; k[1, 0, 1, 0] = 1.0
    v = t64([[1.0, 0.0]], [[0.0, 2.0]])
    o = plain.differential_heads(q, k, v, 1.0, None, 0.5, 0.0, 0.0)
    assert torch.allclose(o[1, 0], t64(1.0, -1.0))
    assert torch.allclose(o[0, 0], t64(math.sqrt(2.0), 0.0))                                # the first token sees only itself: (1 - lambda) v0
    o = plain.differential_heads(q, k, v, 1.0, 1, 0.5, 0.0, 0.0)                            # a window of 1: (1 - lambda) v1
    assert torch.allclose(o[1, 0], t64(0.0, math.sqrt(2.0)))


def test_plain_routing_by_hand():
    """Logits ln(1, 3, 4, 2): scores 0.1, 0.3, 0.4, 0.2.  Corrections turn the choice to experts 0 and 3; the weights stay 0.1 and 0.2.  With
    two experts and two that pass their input on, 3 is one of the latter."""
    w = {"p.router": torch.log(t64([1.0], [3.0], [4.0], [2.0])), "p.correction": t64(0.55, 0.0, -0.3, 0.4),
         "p.e0.gate": t64([2.0]), "p.e0.up": t64([3.0]), "p.e0.down": t64([1.0]),
         "p.shared.gate": t64([1.0]), "p.shared.up": t64([1.0]), "p.shared.down": t64([5.0]), "p.shared.sg": t64([0.0])}
    mlp = {"router": {"experts": 2, "identity": 2, "top": 2}}
    h = t64([1.0])
    got = plain.route(h, mlp, w, "p.")[0]
    assert [e for e, _ in got] == [0, 3] and abs(float(got[0][1]) - 0.1) < 1e-12 and abs(float(got[1][1]) - 0.2) < 1e-12
    silu = lambda z: z / (1 + math.exp(-z))
    assert abs(float(plain.moe_ff(h, mlp, w, "p.")) - (0.1 * silu(2.0) * 3.0 + 0.2)) < 1e-12
    mlp["shared"] = {"ff": 1}
    assert abs(float(plain.moe_ff(h, mlp, w, "p.")) - (0.1 * silu(2.0) * 3.0 + 0.2 + 0.5 * 5.0 * silu(1.0))) < 1e-12


def test_plain_feed_forward_norm_and_parallel_sum_by_hand():
    w = {"p.up": t64([1.0], [-1.0]), "p.down": t64([1.0, 10.0])}
    assert float(plain.dense_ff(t64([3.0]), w, "p.")) == 9.0
    assert torch.allclose(plain.layer_norm(t64([1.0, 3.0]), t64(2.0, 2.0), t64(0.5, -0.5), 0.0), t64([-1.5, 1.5]))
    cfg = CONFIGS["R4"]
    w = {n: t.double() for n, t in make_weights(cfg, 2).items()}
    with torch.no_grad():
        x, after = plain.hidden_states(cfg, w, [3, 9, 27, 81, 5], keep_layers=True)
        h = plain.layer_norm(after[1], w["l1.norm1"], w["l1.norm1.b"], 1e-5)                # layer 2 runs layer 1's tensors on the new stream
        y = plain.attention_mixer(h, cfg["layers"][1]["mixer"], w, "l1.mix.", 1e-5) + plain.dense_ff(h, w, "l1.mlp.")
    assert torch.allclose(after[2], after[1] + y) and torch.equal(after[-1], x)


def test_plain_prefix_does_not_depend_on_what_follows():
    cfg = CONFIGS["R1"]
    w = {n: t.double() for n, t in make_weights(cfg, 3).items()}
    toks = torch.randint(0, cfg["vocab"], (60,), generator=torch.Generator().manual_seed(1)).tolist()
    with torch.no_grad():
        a, b = plain.logits(cfg, w, toks), plain.logits(cfg, w, toks[:47])
    assert torch.allclose(a[:47], b, atol=1e-10)
