"""Razelorn on the GPU against the plain implementation: each mechanism's kernel alone on inputs that show a fault, and the whole model
through the library's step function, cache, scheduler and entry points, in both dtypes, for every way of cutting requests into steps."""
from __future__ import annotations

from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_razelorn as plain
import replay
from conftest import write_model
from razelorn_models import CONFIGS, make_weights, plain_logits, requests_for

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
CASES = [(n, d) for n in sorted(CONFIGS) for d in ("float32", "bfloat16")]
LENGTHS = {"R1": [1, 2, 3, 47, 72, 141, 64, 5], "R2": [65, 1, 150, 9, 33, 2], "R3": [3, 129, 31, 64, 1, 70], "R4": [4, 1, 290, 17, 66, 135],
           "R5": [2, 131, 1, 64, 65, 19]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """{(config, dtype): (engine, cfg, weights, folder)}."""
    from pico_engine.engine.engine import Engine
    root = tmp_path_factory.mktemp("razelorn")
    out = {}
    for k, (name, cfg) in enumerate(sorted(CONFIGS.items())):
        for dtype in DTYPES:                              # bfloat16 runs get corrections that rounding cannot turn
            weights = make_weights(cfg, 90 + k, steady_routing=dtype == "bfloat16")
            folder = write_model(root / f"{name}-{dtype}", cfg, weights)
            out[(name, dtype)] = (Engine(folder, dtype=dtype), cfg, weights, folder)
    return out


def compare(got, cfg, w, reqs, dtype, what, only_got=False):
    """Against the plain logits.  float32: every place, by the rule of the engine tests.  bfloat16: none may be off by more than a tenth of
    the logits' size, and at most one in fifty by more than the engine tests' 4e-2 (a head whose maps nearly cancel is brought to full
    size by its norm and carries its rounding along)."""
    close = set()
    want = plain_logits(cfg, w, reqs, close)
    if only_got:
        want = {k: v for k, v in want.items() if k in got}
    if dtype != "bfloat16":
        return replay.compare(got, want, dtype, what)
    assert set(got) == set(want), (what, sorted(set(want) - set(got))[:5], sorted(set(got) - set(want))[:5])
    assert not close & set(want)
    over = []
    for key in sorted(want, key=lambda k: (str(k[0]), k[1])):
        scale = max(1.0, float(np.abs(want[key]).max()))
        err = float(np.abs(np.asarray(got[key], dtype=np.float64) - want[key]).max()) / scale
        assert err <= 1e-1, f"{what}: request {key[0]!r} position {key[1]}: max error {err:.3e} of the logits' size {scale:.3f}"
        if err > 4e-2:
            over.append((key, round(err, 4)))
    assert len(over) <= max(1, len(want) // 50), (what, len(over), len(want), over[:8])


def check(models, name, dtype, steps, reqs, what):
    eng, cfg, w, _ = models[(name, dtype)]
    compare(replay.run_in_process(eng, steps), cfg, w, reqs, dtype, what)


# ------------------------------------------------------------------ the whole model, every way of cutting

@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_prompts_and_first_tokens(models, name, dtype):
    reqs = requests_for(CONFIGS[name], LENGTHS[name], 1)
    check(models, name, dtype, replay.whole(reqs), reqs, "whole")


@pytest.mark.parametrize("name,dtype", CASES)
def test_prefill_against_token_by_token(models, name, dtype):
    """Every request again with its last tokens one at a time (the shortest ones entirely), 100 for the long ones: the windows pass over
    decoded tokens and pages behind them are given back."""
    reqs = requests_for(CONFIGS[name], LENGTHS[name], 2)
    check(models, name, dtype, replay.tail(reqs, 100), reqs, "tail")


@pytest.mark.parametrize("name,dtype", CASES)
def test_prompts_in_portions(models, name, dtype):
    """Portions of unequal sizes, then portions of two, three and five tokens and single tokens in turn."""
    cfg = CONFIGS[name]
    reqs = requests_for(cfg, LENGTHS[name], 3)
    check(models, name, dtype, replay.pieces(reqs), reqs, "pieces")
    small = requests_for(cfg, [23, 11, 70], 4)
    plan = {}
    for i, (r, toks) in enumerate(small.items()):
        cuts, left, k = [], len(toks), i
        while left:
            c = min(left, (2, 3, 1, 2, 5)[k % 5])
            cuts.append(c); left -= c; k += 1
        plan[r] = (i, cuts)
    check(models, name, dtype, replay.scheduled(small, plan), small, "small portions")


@pytest.mark.parametrize("name,dtype", CASES)
@pytest.mark.parametrize("batch_size,fraction", [(3, 0.5), (8, 0.9)])
def test_unequal_batches_reuse_slots_and_pages(models, name, dtype, batch_size, fraction):
    """Batches one after another in a cache sized for one: slots and pages are used again, and a request's logits do not depend on its
    neighbours (compared with the plain run of each alone)."""
    reqs = requests_for(CONFIGS[name], LENGTHS[name] + LENGTHS[name][::-1], 5)
    check(models, name, dtype, replay.batched(reqs, batch_size, fraction), reqs, "batched")


@pytest.mark.parametrize("name,dtype", CASES)
def test_mixed_steps(models, name, dtype):
    """Steps that carry a fresh prompt, a later portion of another and single tokens side by side."""
    reqs = requests_for(CONFIGS[name], LENGTHS[name], 6)
    check(models, name, dtype, replay.mixed(reqs), reqs, "mixed")


@pytest.mark.parametrize("name,dtype", [("R1", "float32"), ("R1", "bfloat16"), ("R4", "bfloat16"), ("R3", "float32")])
def test_batches_of_more_rows_than_the_decode_products_fuse(models, name, dtype):
    reqs = requests_for(CONFIGS[name], [3 + (7 * i) % 23 for i in range(20)], 13)
    check(models, name, dtype, replay.batched(reqs, 20, 0.5), reqs, "twenty rows")


@pytest.mark.parametrize("name,dtype", [("R1", "float32"), ("R3", "float32"), ("R4", "float32"), ("R4", "bfloat16")])
def test_long_decoding(models, name, dtype):
    """300 tokens one by one from a one-token prompt."""
    reqs = requests_for(CONFIGS[name], [301], 12)
    check(models, name, dtype, replay.tail(reqs, 300), reqs, "long decoding")


def test_a_freed_slot_starts_from_nothing(models):
    eng, cfg, w, _ = models[("R1", "float32")]
    reqs = requests_for(cfg, [40, 6], 8)
    steps = [{"step": 0, "entries": [{"id": "r0", "tokens": reqs["r0"], "want": [39]}], "end": ["r0"]},
             {"step": 1, "entries": [{"id": "r1", "tokens": reqs["r1"], "want": list(range(6))}], "end": ["r1"]}]
    got = replay.run_in_process(eng, steps, max_tokens=64)
    compare(got, cfg, w, reqs, "float32", "slot reuse", only_got=True)


@pytest.mark.parametrize("name", ["R1", "R3", "R4"])
@pytest.mark.parametrize("use_graph", [False, True])
def test_greedy_generation_through_the_entry_point(models, name, use_graph):
    """Engine.generate (scheduler, batches, captured steps) against the plain greedy loop; with graphs three times over, so that prompt
    steps are captured and replayed."""
    eng, cfg, w, _ = models[(name, "float32")]
    w64 = {n: t.double() for n, t in w.items()}
    prompts = list(requests_for(cfg, [5, 1, 19, 66], 9).values())
    news = [12, 20, 7, 9]
    with torch.no_grad():
        want = [plain.greedy(cfg, w64, p, n) for p, n in zip(prompts, news)]
    for _ in range(3 if use_graph else 1):
        assert eng.generate(prompts, max_tokens=news, temperature=0.0, use_graph=use_graph, stop_token_ids=[]) == want


@pytest.mark.parametrize("name", ["R3", "R4"])
def test_bfloat16_generation_with_graphs_matches_eager(models, name):
    eng, cfg, w, _ = models[(name, "bfloat16")]
    prompts = list(requests_for(cfg, [7, 30, 2], 11).values())
    a = eng.generate(prompts, max_tokens=10, temperature=0.0, use_graph=False, stop_token_ids=[])
    for _ in range(3):
        assert eng.generate(prompts, max_tokens=10, temperature=0.0, use_graph=True, stop_token_ids=[]) == a


def test_sublayers_apart_give_what_they_give_on_joined_products(models):
    """The same model with its sublayers run one after the other instead of on shared products."""
    from pico_engine.engine.engine import Engine
    from pico_engine.parts.joined import JoinedSublayers
    for name, dtype in (("R1", "float32"), ("R4", "bfloat16"), ("R3", "float32")):
        _, cfg, w, folder = models[(name, dtype)]
        take = JoinedSublayers.take_tensors
        JoinedSublayers.take_tensors = lambda self, get: None
        try:
            eng = Engine(folder, dtype=dtype)
        finally:
            JoinedSublayers.take_tensors = take
        assert not any(l.joined is not None and l.joined.active for l in eng.model.layers)
        assert any(l.joined is not None and l.joined.active for l in models[(name, dtype)][0].model.layers)
        reqs = requests_for(cfg, [30, 3, 75], 14)
        compare(replay.run_in_process(eng, replay.tail(reqs, 10)), cfg, w, reqs, dtype, "apart")


def test_trace_replay_program(models, tmp_path):
    eng, cfg, w, folder = models[("R2", "float32")]
    reqs = requests_for(cfg, [40, 3, 77], 10)
    steps = replay.batched(reqs, 3, 0.6)
    got = replay.run_binary(folder, "float32", steps, str(tmp_path / "out"), cfg["vocab"])
    compare(got, cfg, w, reqs, "float32", "bin/trace_run")


def test_command_line_generates(models):
    import json, subprocess, sys
    eng, cfg, w, folder = models[("R1", "float32")]
    out = subprocess.run([sys.executable, "-m", "pico_engine", folder, "--prompt", "5,17,3", "--max-tokens", "6", "--temperature", "0",
                          "--dtype", "float32"], capture_output=True, text=True, cwd=replay.ROOT, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    line = [l for l in out.stdout.splitlines() if l.startswith("{")][-1]
    with torch.no_grad():
        assert json.loads(line)["output"] == plain.greedy(cfg, {n: t.double() for n, t in w.items()}, [5, 17, 3], 6)


def test_identity_experts_gates_and_lambdas_count(models, tmp_path):
    """Turning the corrections so that only identity experts are chosen changes the logits as the plain model's do; so do the shared
    expert's gate and the second map's lambda vectors."""
    from pico_engine.engine.engine import Engine
    _, cfg, w, _ = models[("R1", "float32")]
    reqs = requests_for(cfg, [20, 5], 3)
    base = None
    for tag, name, change in (("plain", None, None), ("identity", "l0.mlp.correction", lambda t: torch.cat([t[:6] - 8, t[6:]])),
                              ("gate", "l0.mlp.shared.sg", lambda t: t + 1.0), ("lambda", "l0.mix.lq2", lambda t: t * 3.0)):
        w2 = dict(w)
        if name:
            w2[name] = change(w[name]).to(torch.bfloat16).float()       # (values as they are stored)
        eng = Engine(write_model(tmp_path / tag, cfg, w2), dtype="float32")
        got = replay.run_in_process(eng, replay.whole(reqs))
        compare(got, cfg, w2, reqs, "float32", tag)
        if base is None:
            base = got
        else:
            assert max(np.abs(base[k] - got[k]).max() for k in got) > 1e-2, tag


# ------------------------------------------------------------------ differential attention alone

def run_maps(q, k, v, dt, spans, window, scale, lam, diff, eps, side_col=0, pad_cols=0, first_page=1):
    """``kernels.attention_maps`` for the query positions of ``spans`` (each a step of one sequence); q [n, H, 2, D], k [n, G, 2, D], v [n, G, Dv].
    Returns (heads [n, H, Dv], the columns beside them)."""
    from pico_engine.ops import kernels
    n, H, _, D = q.shape
    G, Dv = k.shape[1], v.shape[2]
    per = H // G
    pages = (n + 63) // 64
    kp = torch.zeros(pages + first_page, 2 * G, 64, D, dtype=dt)
    vp = torch.zeros(pages + first_page, G, 64, Dv, dtype=dt)
    for p in range(n):
        kp[first_page + p // 64, :, p % 64] = k[p].reshape(2 * G, D).to(dt)
        vp[first_page + p // 64, :, p % 64] = v[p].to(dt)
    kp, vp = kp.cuda(), vp.cuda()
    table = torch.arange(first_page, pages + first_page, dtype=torch.int32).view(1, -1).cuda()
    rows = q.view(n, G, per, 2, D).transpose(2, 3).reshape(n, 2 * H * D)
    rows = torch.cat([rows, torch.full((n, 8 + -2 * H * D % 8), 3.0)], dim=1).to(dt).cuda().contiguous()
    side = torch.full((n, side_col + H * Dv + pad_cols), 7.0, dtype=dt).cuda()
    for a, b in spans:
        ctx = SimpleNamespace(one_token_each=(b - a == 1), scratch={}, lens=[b - a], starts=[a], max_context=b, dtype=dt)
        pos, row = torch.arange(a, b, dtype=torch.int32).cuda(), torch.zeros(b - a, dtype=torch.int32).cuda()
        out = side[a:b].clone()
        kernels.attention_maps(rows[a:b].contiguous(), H, G, D, Dv, kp, vp, table, table.shape[1], pos, row, window, scale, lam, eps, 1.0 - diff, out,
                               side_col, ctx)
        side[a:b] = out
    kernels.check_status(side.device)
    side = side.float().cpu()
    return side[:, side_col: side_col + H * Dv].reshape(n, H, Dv), torch.cat([side[:, :side_col], side[:, side_col + H * Dv:]], dim=1)


KERNELS = [("float32", "1"), ("bfloat16", "1"), ("bfloat16", "mma"), ("bfloat16", "0")]


@pytest.mark.parametrize("dtype,which", KERNELS)
@pytest.mark.parametrize("H,G,D,Dv,window", [(4, 2, 64, 128, None), (3, 1, 64, 64, 70), (2, 2, 48, 96, 65), (6, 2, 32, 24, 33), (5, 1, 40, 72, 129), (17, 1, 80, 136, 64),
                                             (4, 4, 128, 256, 100), (2, 1, 256, 256, 130), (8, 1, 16, 8, None), (3, 1, 12, 10, 20), (2, 1, 24, 120, 1)])
def test_differential_attention(monkeypatch, dtype, which, H, G, D, Dv, window):
    """Random queries, keys and values against the plain function at sizes of every kernel: as one prompt, in portions off the borders of pages
    and runs, and the last tokens one by one; columns beside the heads stay as they were."""
    from pico_engine.ops import kernels
    monkeypatch.setattr(kernels, "DIFF_ATTENTION", which)
    dt, n = DTYPES[dtype], 290
    g = torch.Generator().manual_seed(H * 100 + D)
    q, k, v = ((torch.randn(*s, generator=g)).to(dt).float() for s in ((n, H, 2, D), (n, G, 2, D), (n, G, Dv)))
    scale, lam, diff, eps = 1.2 * D ** -0.5, 0.6, 0.3, 1e-5
    want = plain.differential_heads(q.double(), k.double(), v.double(), scale, window, lam, diff, eps)
    one_map = plain.differential_heads(q.double(), k.double(), v.double(), scale, window, 0.0, diff, eps)
    if window != 1:
        assert (want - one_map).abs().max() > 0.1                       # the second map shows
    tol = 3e-5 if dtype == "float32" else 3e-2
    for spans in ([(0, n)], [(0, 3), (3, 70), (70, 72), (72, 200), (200, n)], [(0, 250)] + [(p, p + 1) for p in range(250, n)]):
        got, beside = run_maps(q, k, v, dt, spans, window, scale, lam, diff, eps, side_col=16, pad_cols=8)
        err = (got.double() - want).abs()
        assert err.max() < tol * float(want.abs().max()), (spans[:2], float(err.max()), (err.amax((1, 2)) > tol).nonzero().view(-1)[:8].tolist())
        assert torch.equal(beside, torch.full_like(beside, 7.0))


@pytest.mark.parametrize("dtype,which", KERNELS)
@pytest.mark.parametrize("H,G,D,Dv,window", [(2, 1, 64, 128, 130), (4, 2, 48, 88, 64), (2, 1, 96, 64, 33), (3, 1, 20, 12, 2), (2, 2, 16, 16, 1), (4, 1, 32, 64, 200)])
def test_window_edges_in_prompt_and_decoding(monkeypatch, dtype, which, H, G, D, Dv, window):
    """One key of one map is made to dominate for the queries that follow it: it must be seen by the query window - 1 places after it and
    not by the next one; with the key on either side of a page border and at a sequence's first places, in each map, in a prompt, in
    portions and token by token."""
    from pico_engine.ops import kernels
    monkeypatch.setattr(kernels, "DIFF_ATTENTION", which)
    dt = DTYPES[dtype]
    for mp in (0, 1):
        for key_at in (0, 1, 63, 64, 127):
            n = key_at + window + 70
            g = torch.Generator().manual_seed(key_at)
            q, k = 0.01 * torch.randn(n, H, 2, D, generator=g), 0.01 * torch.randn(n, G, 2, D, generator=g)
            v = torch.randn(n, G, Dv, generator=g)
            v[:, :, 0] = 0.0
            k[key_at, :, mp] = 0; k[key_at, :, mp, D - 1] = 40.0
            q[:, :, mp, D - 1] = 1.0
            v[key_at] = 0; v[key_at, :, 0] = 8.0                         # its value is a direction nobody else's has
            q, k, v = (t.to(dt).float() for t in (q, k, v))
            want = plain.differential_heads(q.double(), k.double(), v.double(), 1.0, window, 0.8, 0.1, 1e-6)
            last = key_at + window - 1
            assert want[last, :, 0].abs().min() > 0.5 * Dv ** 0.5 and want[last + 1, :, 0].abs().max() < 1e-6
            edge = list(range(max(key_at, last - 2), last + 4))
            for spans in ([(0, n)], [(0, last), (last, last + 2), (last + 2, n)], [(p, p + 1) for p in edge]):
                spans = [s for s in spans if s[0] < s[1]]
                got, _ = run_maps(q, k, v, dt, spans, window, 1.0, 0.8, 0.1, 1e-6)
                at = edge if spans[0][0] == edge[0] and spans[0][1] == edge[0] + 1 and edge[0] > 0 else [p for a, b in spans for p in range(a, b)]
                err = (got.double() - want)[at].abs().max()
                assert err < (1e-3 if dtype == "float32" else 4e-2) * float(want.abs().max()), (mp, key_at, spans[:2], float(err))


@pytest.mark.parametrize("dtype,which", KERNELS)
@pytest.mark.parametrize("far", [0, 1, 63, 64, 65, 447, 1000])
def test_a_key_from_far_back(monkeypatch, dtype, which, far):
    """Without a window one key that matches the last query of one map must come through from any distance; in a prompt and alone."""
    from pico_engine.ops import kernels
    monkeypatch.setattr(kernels, "DIFF_ATTENTION", which)
    dt, n = DTYPES[dtype], 1210
    for H, G, D, Dv in ((2, 1, 64, 128), (2, 2, 80, 40)):
        for mp in (0, 1):
            g = torch.Generator().manual_seed(far)
            q, k, v = 0.01 * torch.randn(n, H, 2, D, generator=g), 0.01 * torch.randn(n, G, 2, D, generator=g), torch.randn(n, G, Dv, generator=g)
            v[:, :, 0] = 0.0
            k[far, :, mp] = 0; k[far, :, mp, D - 1] = 40.0
            q[-1, :, mp] = 0; q[-1, :, mp, D - 1] = 1.0
            v[far] = 0; v[far, :, 0] = 8.0
            q, k, v = (t.to(dt).float() for t in (q, k, v))
            for spans in ([(0, n)], [(n - 1, n)]):
                got, _ = run_maps(q, k, v, dt, spans, None, 1.0, 0.8, 0.0, 1e-6)
                sign = 1.0 if mp == 0 else -1.0
                assert (got[-1, :, 0] * sign).min() > 0.97 * Dv ** 0.5, (far, mp, got[-1, :, 0])


@pytest.mark.parametrize("which", ["1", "mma"])
@pytest.mark.parametrize("H,G,D,Dv,window", [(4, 1, 64, 128, None), (2, 1, 64, 128, 600), (4, 2, 56, 88, 300), (2, 1, 128, 128, None)])
def test_long_prompts_in_bfloat16(monkeypatch, which, H, G, D, Dv, window):
    """1,100 tokens whole, in portions off the borders, and with the last 100 one by one (whose keys a cluster's blocks share)."""
    from pico_engine.ops import kernels
    monkeypatch.setattr(kernels, "DIFF_ATTENTION", which)
    dt, n = torch.bfloat16, 1100
    g = torch.Generator().manual_seed(D)
    q, k, v = ((torch.randn(*s, generator=g)).to(dt).float() for s in ((n, H, 2, D), (n, G, 2, D), (n, G, Dv)))
    scale = 2.0 * D ** -0.5
    want = plain.differential_heads(q.double(), k.double(), v.double(), scale, window, 0.4, 0.2, 1e-5)
    for spans in ([(0, n)], [(0, 130), (130, 133), (133, 517), (517, n)], [(0, 1000)] + [(p, p + 1) for p in range(1000, n)]):
        got, _ = run_maps(q, k, v, dt, spans, window, scale, 0.4, 0.2, 1e-5)
        err = (got.double() - want).abs()
        assert err.max() < 3e-2 * float(want.abs().max()), (spans[:2], float(err.max()))


# ------------------------------------------------------------------ the other kernels alone

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,Gv,D,Dv,rot,normed", [(4, 2, 1, 64, 128, 48, True), (6, 4, 2, 48, 24, 16, True), (3, 2, 1, 12, 10, 10, True), (2, 2, 1, 80, 136, 80, True),
                                                    (5, 1, 1, 256, 16, 256, True), (4, 4, 4, 16, 8, 0, True), (2, 2, 1, 40, 8, 6, False), (34, 2, 1, 8, 8, 4, True)])
def test_norm_rotation_and_store(dtype, H, G, Gv, D, Dv, rot, normed):
    """Every query and key row normed by itself (one row far larger than the others must not show in them), halves turned up to position 4,999,
    keys and values at their places in the cache, the columns behind untouched."""
    from pico_engine.ops import kernels
    dt = DTYPES[dtype]
    T, ld = 5, H * D + G * D + Gv * Dv + 8 + -(H * D + G * D + Gv * Dv) % 8
    g = torch.Generator().manual_seed(H + D)
    x = torch.randn(T, ld, generator=g)
    x[1, :D] *= 50.0
    x = x.to(dt).float()
    qw, kw = (1.0 + 0.3 * torch.randn(D, generator=g)).to(dt).float(), (1.0 + 0.3 * torch.randn(D, generator=g)).to(dt).float()
    pos = torch.tensor([0, 63, 64, 1000, 4999])
    freqs = plain.frequencies(rot, 500.0, {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 200}) if rot else []
    kp, vp = torch.zeros(160, G, 64, D, dtype=dt).cuda(), torch.zeros(160, Gv, 64, Dv, dtype=dt).cuda()
    perm = torch.randperm(80, generator=g).to(torch.int32) + 7
    table = torch.stack([perm, perm + 60]).contiguous().cuda()
    rows = torch.tensor([0, 1, 0, 1, 0], dtype=torch.int32)
    proj = x.to(dt).cuda()
    kernels.heads_norm_store(proj, H, G, Gv, D, Dv, qw.to(dt).cuda() if normed else None, kw.to(dt).cuda() if normed else None, 1e-4,
                             torch.tensor(freqs, dtype=torch.float32).cuda() if rot else None, rot, pos.to(torch.int32).cuda(), rows.cuda(), kp, vp, table, 80)
    tol = 2e-4 if dtype == "float32" else 2e-2          # (float32 angles at position 4,999)
    for t in range(T):
        heads = x[t, :(H + G) * D].double().view(H + G, D)
        if normed:
            heads = plain.rms_unit(heads, 1e-4) * torch.cat([qw.double().expand(H, D), kw.double().expand(G, D)])
        if rot:
            h = rot // 2
            a = torch.tensor([float(pos[t]) * f for f in freqs], dtype=torch.float64)
            u, v = heads[:, :h].clone(), heads[:, h:rot].clone()
            heads = heads.clone()
            heads[:, :h], heads[:, h:rot] = u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()
        size = max(1.0, float(heads.abs().max()))
        assert (proj[t, :H * D].cpu().double().view(H, D) - heads[:H]).abs().max() < tol * size
        page, at = int(table[rows[t], int(pos[t]) // 64]), int(pos[t]) % 64
        assert (kp[page, :, at].cpu().double() - heads[H:]).abs().max() < tol * size
        assert torch.equal(vp[page, :, at].cpu().float().reshape(-1), x[t, (H + G) * D:(H + G) * D + Gv * Dv])
        assert torch.equal(proj[t, (H + G) * D:].cpu().float(), x[t, (H + G) * D:])
    assert int((kp != 0).any(-1).sum()) <= T * G and int((vp != 0).any(-1).sum()) <= T * Gv


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,K,E,I,gate,top", [(3, 80, 6, 3, True, 3), (9, 50, 3, 2, False, 1), (700, 64, 8, 0, True, 2), (601, 128, 12, 4, True, 2), (2, 4096, 5, 1, False, 6),
                                              (1, 72, 200, 56, True, 7), (650, 3584, 8, 2, True, 2)])
def test_routing_of_normed_rows(dtype, T, K, E, I, gate, top):
    """Weights, the chosen, the gate's column and the share that is passed on, for few tokens (a block each) and many (four a block), with
    corrections that turn choices; zeros where nothing was chosen."""
    from pico_engine.ops import kernels
    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(K + T)
    h = torch.randn(T, K, generator=g).to(dt).float()
    router = (torch.randn(E + I + gate, K, generator=g) * 1.5 * K ** -0.5).to(dt).float()
    corr = torch.randperm(E + I, generator=g).float() * 0.01 + (torch.rand(E + I, generator=g) < 0.3).float() * 1.1
    ids = torch.empty(T, top, dtype=torch.int32).cuda()
    got = kernels.route_rows(h.to(dt).cuda(), router.to(dt).cuda(), E + I, E, top, corr.cuda(), gate, 1.0, ids).cpu().double()
    w = {"p.router": router[:E + I].double(), "p.correction": corr.double()}
    plain.ROUTER_GAPS = []
    want = plain.route(h.double(), {"router": {"top": top}}, w, "p.")
    gaps, plain.ROUTER_GAPS = plain.ROUTER_GAPS[0], None
    assert got.shape == (T, E + gate + (I > 0))
    clear = 0
    for t in range(T):
        chosen = [e for e, _ in want[t]]
        if float(gaps[t]) < 1e-5:
            continue
        clear += 1
        assert sorted(ids[t].tolist()) == sorted(chosen)
        row = torch.zeros(E + gate + (I > 0), dtype=torch.float64)
        for e, s in want[t]:
            row[e if e < E else -1] += float(s)
        if gate:
            row[E] = float(plain.sigmoid(router[-1].double() @ h[t].double()))
        assert (got[t] - row).abs().max() < 2e-5
        assert all(float(got[t, e]) == 0.0 for e in range(E) if e not in chosen)
    assert clear > 0.9 * T and len({tuple(ids[t].tolist()) for t in range(T)}) > (1 if T > 3 else 0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,W", [(1, 50), (5, 80), (300, 896), (7, 3584), (3, 5000), (2, 4096)])
def test_sum_and_layer_norm(dtype, T, W):
    """x += y + a * rows in float32, in place, and the layer norm of the new rows; each part alone as well."""
    from pico_engine.ops import kernels
    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(W)
    x, y, r = torch.randn(T, W, generator=g) * 3 + 1, torch.randn(T, W, generator=g), torch.randn(T, W, generator=g).to(dt).float()
    a = torch.rand(T, 3, generator=g)
    a[T // 2, 1] = 0.0
    w, b = 1 + 0.2 * torch.randn(W, generator=g), torch.randn(W, generator=g)
    for yy in (y, y.to(torch.bfloat16).float(), None):
        for rows in (True, False):
            want = x.double() + (0 if yy is None else yy.double()) + (a[:, 1:2].double() * r.double() if rows else 0)
            xs, aw = x.clone().cuda(), a.cuda()
            yc = None if yy is None else (yy.cuda() if yy is y else yy.to(torch.bfloat16).cuda())
            out = kernels.add_layernorm(xs, yc, (w.cuda(), b.cuda(), 1e-5), dt, *((r.to(dt).cuda(), aw[:, 1]) if rows else (None, None)))
            assert (xs.cpu().double() - want).abs().max() < 1e-5
            ln = plain.layer_norm(want, w.double(), b.double(), 1e-5)
            assert (out.cpu().double() - ln).abs().max() < (2e-5 if dtype == "float32" else 2e-2) * float(ln.abs().max())
            xs = x.clone().cuda()
            assert kernels.add_layernorm(xs, yc, None, None, *((r.to(dt).cuda(), aw[:, 1]) if rows else (None, None))) is None
            assert (xs.cpu().double() - want).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,E,F,S,gated", [(3, 4, 24, 40, True), (5, 3, 13, 11, True), (70, 8, 32, 0, True), (4, 1, 160, 0, False), (2, 2, 12, 0, False)])
def test_activation_into_the_side_rows(dtype, T, E, F, S, gated):
    """Hidden units of weighted experts from a column range into another, exact zeros (and no reads: their inputs are NaN) for unused
    experts, columns beside them untouched."""
    from pico_engine.ops import kernels
    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(F)
    I, n_groups = E * F + S, E + (1 if S else 0)
    col, out_col = 16, 24
    src = torch.randn(T, col + (2 if gated else 1) * I + -((2 if gated else 1) * I) % 8 + 8, generator=g).to(dt).float()
    weights = torch.rand(T, n_groups + 1, generator=g)
    weights[:, 0] = 0.0
    use = E > 1
    if use:
        src[:, col: col + F] = float("nan")
    out = torch.full((T, out_col + I + -I % 8 + 8), 7.0, dtype=dt).cuda()
    kernels.side_act(src.to(dt).cuda(), col, col + I if gated else -1, I, "silu" if gated else "relu2", out, out_col, weights.cuda() if use else None, F, n_groups)
    out = out.float().cpu()
    for c in range(I):
        z = src[:, col + c].double()
        f = z * plain.sigmoid(z) * src[:, col + I + c].double() if gated else torch.clamp(z, min=0) ** 2
        if use:
            grp = min(c // F, n_groups - 1)
            f = torch.zeros(T).double() if grp == 0 else f * weights[:, grp].double()
        assert (out[:, out_col + c].double() - f).abs().max() < (1e-5 if dtype == "float32" else 2e-2) * max(1.0, float(f.abs().max())), c
    assert torch.equal(out[:, :out_col], torch.full((T, out_col), 7.0)) and torch.equal(out[:, out_col + I:], torch.full_like(out[:, out_col + I:], 7.0))
