"""Lefilorn on the GPU against the plain implementation: each mechanism's kernel alone on inputs that show a fault, and the whole
model through the library's step function, cache, scheduler and entry points, in both dtypes, for every way of cutting requests
into steps."""
from __future__ import annotations

from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_lefilorn as plain
import replay
from conftest import write_model
from lefilorn_models import CONFIGS, SEEDS, make_weights, plain_logits, requests_for

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
CASES = [(n, d) for n in sorted(CONFIGS) for d in ("float32", "bfloat16")]
LENGTHS = {"L1": [1, 2, 3, 47, 70, 131, 64, 5], "L2": [65, 1, 110, 9, 33, 2], "L3": [4, 1, 290, 17, 66, 135], "L4": [3, 129, 31, 64, 1, 70],
           "L5": [2, 230, 1, 66, 40], "L6": [25, 1, 100]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """{(config, dtype): (engine, cfg, weights, folder)}."""
    from pico_engine.engine.engine import Engine
    root = tmp_path_factory.mktemp("lefilorn")
    out = {}
    for name, cfg in sorted(CONFIGS.items()):
        weights = make_weights(cfg, SEEDS[name])
        folder = write_model(root / name, cfg, weights)
        for dtype in DTYPES:
            out[(name, dtype)] = (Engine(folder, dtype=dtype), cfg, weights, folder)
    return out


def compare(got, cfg, w, reqs, dtype, what, only_got=False):
    """Against the plain logits.  float32: every place, by the rule of the engine tests.  bfloat16: none may be off by more than a tenth
    of the logits' size, and at most one in fifty by more than the engine tests' 4e-2 (every head of the linear branch is divided by
    its own root mean square, so a head whose output is small carries its rounding at full size)."""
    want = plain_logits(cfg, w, reqs)
    if only_got:
        want = {k: v for k, v in want.items() if k in got}
    if dtype != "bfloat16":
        return replay.compare(got, want, dtype, what)
    assert set(got) == set(want), (what, sorted(set(want) - set(got))[:5], sorted(set(got) - set(want))[:5])
    over = []
    for key in sorted(want, key=lambda k: (str(k[0]), k[1])):
        scale = max(1.0, float(np.abs(want[key]).max()))
        err = float(np.abs(np.asarray(got[key], dtype=np.float64) - want[key]).max()) / scale
        assert err <= 1e-1, f"{what}: request {key[0]!r} position {key[1]}: max error {err:.3e} of the logits' size {scale:.3f}"
        if err > 4e-2:
            over.append((key, round(err, 4)))
    assert len(over) <= max(1, len(want) // 50), (what, over[:8])


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
    """Every request again with its last tokens one at a time (the shortest ones entirely), 100 for the long ones: windows pass over
    decoded tokens, pages between the kept ones and the window are given back, states are carried from token to token."""
    reqs = requests_for(CONFIGS[name], LENGTHS[name], 1)
    check(models, name, dtype, replay.tail(reqs, 100), reqs, "tail")


@pytest.mark.parametrize("name,dtype", CASES)
def test_prompts_in_portions(models, name, dtype):
    """Portions of unequal sizes, then portions of two, three and five tokens and single tokens in turn: every portion starts inside
    its sequence from the cache pages and the state the portion before it left."""
    cfg = CONFIGS[name]
    reqs = requests_for(cfg, LENGTHS[name], 1)
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
    """Batches one after another in a cache sized for one: slots, pages and state rows are used again, and a request's logits do not
    depend on its neighbours (compared with the plain run of each alone)."""
    reqs = requests_for(CONFIGS[name], LENGTHS[name] + LENGTHS[name][::-1], 5)
    check(models, name, dtype, replay.batched(reqs, batch_size, fraction), reqs, "batched")


@pytest.mark.parametrize("name,dtype", CASES)
def test_mixed_steps(models, name, dtype):
    """Steps that carry a fresh prompt, a later portion of another and single tokens side by side."""
    reqs = requests_for(CONFIGS[name], LENGTHS[name], 1)
    check(models, name, dtype, replay.mixed(reqs), reqs, "mixed")


@pytest.mark.parametrize("name,dtype", [("L1", "float32"), ("L1", "bfloat16"), ("L3", "bfloat16"), ("L4", "float32"), ("L5", "bfloat16")])
def test_batches_of_more_rows_than_the_decode_products_fuse(models, name, dtype):
    """Twenty short requests start together and are decoded together: steps of 17 and more rows take the products that prompts take."""
    reqs = requests_for(CONFIGS[name], [3 + (7 * i) % 23 for i in range(20)], 13)
    check(models, name, dtype, replay.batched(reqs, 20, 0.5), reqs, "twenty rows")


@pytest.mark.parametrize("name,dtype", [("L1", "float32"), ("L3", "float32"), ("L3", "bfloat16")])
def test_long_decoding(models, name, dtype):
    """300 tokens one by one from a one-token prompt: windows, kept tokens, pages given back, and states over many steps."""
    reqs = requests_for(CONFIGS[name], [301], 12)
    check(models, name, dtype, replay.tail(reqs, 300), reqs, "long decoding")


def test_a_freed_slot_starts_from_nothing(models):
    """A sequence that takes over a slot must see neither the keys nor the matrix states left there."""
    eng, cfg, w, _ = models[("L1", "float32")]
    reqs = requests_for(cfg, [40, 6], 8)
    steps = [{"step": 0, "entries": [{"id": "r0", "tokens": reqs["r0"], "want": [39]}], "end": ["r0"]},
             {"step": 1, "entries": [{"id": "r1", "tokens": reqs["r1"], "want": list(range(6))}], "end": ["r1"]}]
    got = replay.run_in_process(eng, steps, max_tokens=64)
    compare(got, cfg, w, reqs, "float32", "slot reuse", only_got=True)


@pytest.mark.parametrize("name", ["L1", "L3", "L5"])
@pytest.mark.parametrize("use_graph", [False, True])
def test_greedy_generation_through_the_entry_point(models, name, use_graph):
    """Engine.generate (scheduler, batches, captured prompt and decode steps) against the plain greedy loop; twice, so that a prompt
    step of these sizes is captured and replayed."""
    eng, cfg, w, _ = models[(name, "float32")]
    w64 = {n: t.double() for n, t in w.items()}
    prompts = list(requests_for(cfg, [5, 1, 19, 66], 9).values())
    news = [12, 20, 7, 9]
    with torch.no_grad():
        want = [plain.generate(p, w64, cfg, n)[len(p):] for p, n in zip(prompts, news)]
    for _ in range(3 if use_graph else 1):
        assert eng.generate(prompts, max_tokens=news, temperature=0.0, use_graph=use_graph, stop_token_ids=[]) == want


@pytest.mark.parametrize("name", ["L3", "L4"])
def test_bfloat16_generation_with_graphs_matches_eager(models, name):
    eng, cfg, w, _ = models[(name, "bfloat16")]
    prompts = list(requests_for(cfg, [7, 30, 2], 11).values())
    a = eng.generate(prompts, max_tokens=10, temperature=0.0, use_graph=False, stop_token_ids=[])
    b = eng.generate(prompts, max_tokens=10, temperature=0.0, use_graph=True, stop_token_ids=[])
    assert a == b


@pytest.mark.parametrize("name,dtype", [("L1", "float32"), ("L2", "float32"), ("L3", "bfloat16")])
def test_branches_apart_give_what_branches_together_give(models, name, dtype, monkeypatch):
    """The same model whose branches do not share their products (each mixer by itself, its outputs scaled and summed)."""
    from pico_engine.engine.engine import Engine
    from pico_engine.parts import LinearAttention
    _, cfg, w, folder = models[(name, dtype)]
    monkeypatch.setattr(LinearAttention, "can_share", lambda self: False)
    eng = Engine(folder, dtype=dtype)
    assert not eng.model.layers[0].mixer.shared and models[(name, dtype)][0].model.layers[0].mixer.shared
    reqs = requests_for(cfg, LENGTHS[name], 1)
    compare(replay.run_in_process(eng, replay.tail(reqs, 20)), cfg, w, reqs, dtype, "apart")


def test_trace_replay_program(models, tmp_path):
    """``--max-tokens`` counts tokens: the partly filled pages of three requests need no allowance of the caller's."""
    eng, cfg, w, folder = models[("L2", "float32")]
    reqs = requests_for(cfg, [40, 3, 77], 10)
    steps = replay.batched(reqs, 3, 0.6)
    got = replay.run_binary(folder, "float32", steps, str(tmp_path / "out"), cfg["vocab"], max_tokens=120)
    compare(got, cfg, w, reqs, "float32", "bin/trace_run")


def test_command_line_generates(models):
    import json, subprocess, sys
    eng, cfg, w, folder = models[("L1", "float32")]
    out = subprocess.run([sys.executable, "-m", "pico_engine", folder, "--prompt", "5,17,3", "--max-tokens", "6", "--temperature", "0",
                          "--dtype", "float32"], capture_output=True, text=True, cwd=replay.ROOT, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    line = [l for l in out.stdout.splitlines() if l.startswith("{")][-1]
    with torch.no_grad():
        assert [5, 17, 3] + json.loads(line)["output"] == plain.generate([5, 17, 3], {n: t.double() for n, t in w.items()}, cfg, 6)


# ------------------------------------------------------------------ norm over all heads, rotation, cache write; the linear branch's rotation

def cached(n, G, D, dt, first=2):
    """Empty pages and the table of one sequence whose logical page p is physical page first + p (pages before `first` are others')."""
    pages = (n + 63) // 64
    return torch.zeros(first + pages, G, 64, D, dtype=dt).cuda(), torch.arange(first, first + pages, dtype=torch.int32).view(1, -1).cuda()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("halves", [False, True])
@pytest.mark.parametrize("H,G,D,Dv,rot", [(4, 2, 32, 16, 16), (3, 1, 24, 12, 10), (8, 1, 64, 64, 64), (2, 2, 10, 7, 10), (16, 4, 128, 128, 96),
                                          (70, 2, 128, 24, 8), (5, 1, 40, 40, 0), (1, 1, 256, 8, 256)])
def test_norm_over_all_heads_rotation_and_store(dtype, halves, H, G, D, Dv, rot):
    from pico_engine.ops import kernels
    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(H * 7 + D)
    pos = [0, 1, 63, 64, 130, 4999]
    n, extra = len(pos), 8 - ((H + G) * D + G * Dv) % 8 + 8
    rows = torch.randn(n, (H + G) * D + G * Dv + extra, generator=g).to(dt)
    rows[:, :D] *= 3.0                                       # one head larger than the others: a norm head by head would hide it
    qw, kw = (1.0 + 0.3 * torch.randn(m, generator=g) for m in (H * D, G * D))
    base, eps = 10000.0, 0.05
    freq = torch.tensor([base ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float32).cuda() if rot else None
    for normed in (True, False):
        proj = rows.clone().cuda()
        kp, table = cached(5000, G, D, dt)
        vp, _ = cached(5000, G, Dv, dt)
        w = [None, None] if not normed else [t.to(dt).cuda() for t in (qw, kw)]
        kernels.heads_prepare(proj, torch.tensor(pos, dtype=torch.int32).cuda(), torch.zeros(n, dtype=torch.int32).cuda(),
                              kernels.NormedHeads(H, G, D, Dv, w[0], w[1], eps, freq, rot, halves, kp, vp, table, table.shape[1]))
        x = rows.double()
        q, k = x[:, :H * D], x[:, H * D:(H + G) * D]
        if normed:
            q, k = plain.rms_norm(q, w[0].double().cpu(), eps), plain.rms_norm(k, w[1].double().cpu(), eps)
        turn = plain.rotate_halves if halves else plain.rotate_neighbours
        f = (lambda u, heads: torch.cat([turn(u[i:i + 1].view(1, heads, D), rot, base, first=p) for i, p in enumerate(pos)])) if rot else \
            (lambda u, heads: u.view(n, heads, D))
        q, k = f(q, H), f(k, G)
        tol = 1e-2 if dtype == "bfloat16" else 2e-3 * (4999 / 5000)       # position 4,999 times a float32 frequency: the angle is good to 3e-4
        got = proj.double().cpu()
        assert (got[:, :H * D].view(n, H, D) - q).abs().max() < tol * max(1.0, float(q.abs().max()))
        assert (got[:3, :H * D].view(3, H, D) - q[:3]).abs().max() < (1e-2 if dtype == "bfloat16" else 2e-5) * max(1.0, float(q.abs().max()))
        assert (got[:, H * D:(H + G) * D].view(n, G, D) - k).abs().max() < tol * max(1.0, float(k.abs().max()))
        assert torch.equal(got[:, (H + G) * D:], x[:, (H + G) * D:])
        for i, p in enumerate(pos):
            at = (2 + p // 64, slice(None), p % 64)
            assert torch.equal(kp[at].double().cpu().reshape(-1), got[i, H * D:(H + G) * D])
            assert torch.equal(vp[at].double().cpu().reshape(-1), x[i, (H + G) * D:(H + G) * D + G * Dv])
        assert float(kp.float().abs().sum(dim=(1, 3)).count_nonzero()) == n and not kp[:2].any()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("halves", [True, False])
@pytest.mark.parametrize("H,D,rot,before", [(3, 16, 8, 8), (2, 20, 6, 24), (1, 64, 64, 0), (4, 8, 0, 16), (2, 136, 136, 8), (1, 7, 2, 3), (2, 256, 128, 0)])
def test_turned_heads_in_float32(dtype, halves, H, D, rot, before):
    """Queries and keys of a linear attention turned and scaled into float32 rows: not rounded on the way, the product's rows stay."""
    from pico_engine.ops import kernels
    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(D)
    pos = list(range(3, 9)) + [640]
    n = len(pos)
    rows = torch.randn(n, before + 2 * H * D + 5, generator=g).to(dt)
    proj = rows.clone().cuda()
    freq = torch.tensor([200.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float32).cuda() if rot else None
    got = kernels.heads_prepare(proj, torch.tensor(pos, dtype=torch.int32).cuda(), torch.zeros(n, dtype=torch.int32).cuda(), None,
                                kernels.TurnedHeads(H, D, before, before + H * D, freq, rot, halves, 0.25)).double().cpu()
    turn = plain.rotate_halves if halves else plain.rotate_neighbours
    x = rows.double()[:, before:before + 2 * H * D].view(n, 2 * H, D)
    want = torch.cat([turn(x[i:i + 1], rot, 200.0, first=p) for i, p in enumerate(pos)]) if rot else x.clone()
    want[:, H:] *= 0.25
    assert torch.equal(proj.cpu(), rows)
    assert (got.view(n, 2 * H, D) - want).abs().max() < 3e-4
    assert (got.view(n, 2 * H, D)[:6] - want[:6]).abs().max() < 3e-6


# ------------------------------------------------------------------ gates side by side

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [[(64, 0), (48, 16)], [(10, 0), (12, 4), (9, 3)], [(96, 32)], [(2048, 0), (1024, 128)], [(40, 40), (600, 600)], [(30, 10), (64, 0)],
                                   [(8, 8), (16, 0), (12, 12), (20, 4)]])
def test_gated_rows_side_by_side(dtype, sizes):
    from pico_engine.ops import kernels
    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(sum(c for c, _ in sizes))
    n, eps = 37, 0.02
    total = sum(c for c, _ in sizes)
    lead = 16
    gate = torch.randn(n, lead + total + 4, generator=g).to(dt)
    width = (total + 7) // 8 * 8
    jobs, want, at = [], [], lead
    for i, (c, group) in enumerate(sizes):
        f32 = group > 0
        rows = (torch.randn(n, c, generator=g) * (0.1 + torch.rand(n, 1, generator=g))).to(torch.float32 if f32 else dt)
        weight = (1 + 0.2 * torch.randn(group, generator=g)).to(dt) if group and i % 2 else None
        act, scale = ("silu", -0.6) if group else ("sigmoid", 1.7)
        jobs.append(kernels.GatedRows(rows.cuda(), group, None if weight is None else weight.cuda(), eps, at, act, scale))
        z = gate[:, at:at + c].double()
        o = rows.double()
        if group:
            o = plain.unit_rms(o.view(n, c // group, group), eps) * (1 if weight is None else weight.double())
            o = o.reshape(n, c)
        want.append(scale * o * (z * plain.sigmoid(z) if act == "silu" else plain.sigmoid(z)))
        at += c
    got = kernels.gate_heads(jobs, gate.cuda(), width).double().cpu()
    want = torch.cat(want, dim=1)
    assert got.shape == (n, width) and not got[:, total:].any()
    assert (got[:, :total] - want).abs().max() < (8e-3 if dtype == "bfloat16" else 3e-6) * max(1.0, float(want.abs().max()))


# ------------------------------------------------------------------ streams

@pytest.mark.parametrize("S,W", [(1, 48), (2, 72), (3, 192), (4, 1024), (5, 4096), (8, 256), (9, 64), (4, 4104), (2, 50), (32, 33), (3, 12000), (6, 128), (7, 20)])
def test_streams_after_a_sublayer_and_what_the_next_one_reads(S, W):
    """Against the plain functions in float64: from several streams and from the one matrix they all equal at first; with and without a
    sublayer's output; in place and apart; the norm in both dtypes, and the plain sum."""
    from pico_engine.ops import kernels
    g = torch.Generator().manual_seed(S * 1000 + W)
    n, eps = 5, 0.01
    x = torch.randn(n, S, W, generator=g)
    y = torch.randn(n, W, generator=g)
    mix, out, inn = torch.randn(S, S, generator=g), torch.randn(S, generator=g), torch.randn(S, generator=g)
    w = 1 + 0.2 * torch.randn(W, generator=g)
    dev = [t.cuda() for t in (mix, out, inn)]
    for one in (False, True):
        xs = [x[:, 0].double()] * S if one else [x[:, s].double() for s in range(S)]
        for y_dtype in (torch.float32, torch.bfloat16):
            yy = y.to(y_dtype)
            new = plain.streams_out(xs, yy.double(), mix.double(), out.double())
            scale = max(float(t.abs().max()) for t in new)
            src = (x[:, 0].contiguous() if one else x.clone()).cuda()
            dst = torch.full((n, S, W), float("nan")).cuda() if one else src
            for dt, wd in ((torch.float32, w), (torch.bfloat16, w.to(torch.bfloat16))):
                s2, d2 = src.clone(), dst.clone()
                if not one:
                    s2 = d2
                h = kernels.stream_mix(s2, S, d2, yy.cuda(), *dev[:2], dev[2], wd.cuda(), eps, dt)
                want = plain.rms_norm(plain.streams_in(new, inn.double()), wd.double(), eps)
                assert (torch.stack(new, 1) - d2.double().cpu()).abs().max() < 2e-6 * scale * S
                assert (h.double().cpu() - want).abs().max() < (3e-5 if dt == torch.float32 else 1e-2) * max(1.0, float(want.abs().max()))
            total = kernels.stream_mix(src, S, None, yy.cuda(), *dev[:2], out_dtype=torch.float32).double().cpu()
            assert (total - sum(new)).abs().max() < 3e-6 * scale * S * S ** 0.5
        h = kernels.stream_mix(src, S, None, None, in_weights=dev[2], norm_weight=w.cuda(), eps=eps, out_dtype=torch.float32).double().cpu()
        assert (h - plain.rms_norm(plain.streams_in(xs, inn.double()), w.double(), eps)).abs().max() < 3e-5 * max(1.0, float(h.abs().max()))
        assert torch.equal(src.cpu(), x[:, 0] if one else x)                              # nothing pending: the streams stay
        spread = torch.empty(n, S, W).cuda()
        assert kernels.stream_mix(src, S, spread) is None
        assert torch.equal(spread.cpu(), torch.stack([t.float() for t in xs], 1))


def test_the_mix_is_indexed_from_to():
    from pico_engine.ops import kernels
    for W in (8, 7):
        x = torch.zeros(1, 2, W).cuda(); x[0, 0] = 1.0; x[0, 1] = 10.0
        mix = torch.tensor([[1.0, 0.25], [0.0, 2.0]]).cuda()
        kernels.stream_mix(x, 2, x, torch.full((1, W), 100.0).cuda(), mix, torch.tensor([1.0, -1.0]).cuda())
        assert x[0, 0].tolist() == [101.0] * W and x[0, 1].tolist() == [-79.75] * W


# ------------------------------------------------------------------ linear attention on turned rows

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,Dv", [(3, 16, 24), (2, 20, 12), (2, 64, 64), (1, 136, 40), (2, 128, 130), (4, 8, 8), (1, 256, 16)])
def test_recurrence_on_float32_queries_and_keys(dtype, H, D, Dv):
    """Queries and keys in float32 rows of their own, values in the product's rows and dtype: as one prompt in chunks and token by token,
    in portions, and one token at a time; outputs and states.  The float32 entries carry bits that bfloat16 has not."""
    from pico_engine.ops import kernels
    dt = DTYPES[dtype]
    g = torch.Generator().manual_seed(H * 100 + D)
    lens = [1, 64, 65, 130, 2]
    T, B = sum(lens), len(lens)
    qk = torch.randn(T, 2 * H * D, generator=g) * D ** -0.25
    lead = 8
    proj = torch.randn(T, lead + H * Dv + 3, generator=g).to(dt)
    decay = [0.97, 0.5, 1.0, 0.0][:H]
    v = proj[:, lead:lead + H * Dv].double().view(T, H, Dv)
    first = np.concatenate([[0], np.cumsum(lens)])
    want, states = [], []
    for b in range(B):
        sl = slice(first[b], first[b + 1])
        q, k = (qk[sl, i * H * D:(i + 1) * H * D].double().view(-1, H, D) for i in (0, 1))
        want.append(plain.retention(q, k, v[sl], decay))
        S = torch.zeros(H, D, Dv, dtype=torch.float64)
        for t in range(lens[b]):
            S = torch.tensor(decay).double().view(H, 1, 1) * S + k[t][:, :, None] * v[sl][t][:, None, :]
        states.append(S)
    want, states = torch.cat(want), torch.stack(states)
    hd = torch.tensor(decay, dtype=torch.float32).cuda()
    slots = torch.arange(1, B + 1, dtype=torch.int32).cuda()
    for cuts, chunked in (((1.0,), True), ((1.0,), False), ((0.4, 0.75, 1.0), True), ((0.9, 0.95, 1.0), False)):
        state = torch.zeros(B + 2, 5 + H * D * Dv).cuda()
        out, done = torch.zeros(T, H * Dv), [0] * B
        for c in cuts:
            upto = [m if c == cuts[-1] else max(d, int(m * c)) for m, d in zip(lens, done)]
            rows = [b for b in range(B) if upto[b] > done[b]]
            idx = torch.cat([torch.arange(first[b] + done[b], first[b] + upto[b]) for b in rows])
            step = [upto[b] - done[b] for b in rows]
            rf = torch.tensor(np.concatenate([[0], np.cumsum(step)]), dtype=torch.int32).cuda()
            o = kernels.linear_attention(proj[idx].cuda(), 0, H * D, lead, H, D, Dv, state, 5, rf, torch.tensor(step, dtype=torch.int32).cuda(),
                                         slots[torch.tensor(rows).cuda()].contiguous(), chunked, head_decay=hd, qk=qk[idx].cuda())
            out[idx] = o.cpu()
            done = upto
        scale = max(1.0, float(want.abs().max()))
        assert (out.view(T, H, Dv).double() - want).abs().max() < 1e-5 * scale, (cuts, chunked)
        assert (state[1:B + 1, 5:].cpu().view(B, H, D, Dv).double() - states).abs().max() < 1e-5 * max(1.0, float(states.abs().max()))
        assert not state[0].any() and not state[B + 1].any() and not state[:, :5].any()


@pytest.mark.parametrize("far", [0, 1, 63, 64, 65, 447])
@pytest.mark.parametrize("chunked", [True, False])
def test_a_key_from_far_back_survives_the_decay(far, chunked):
    """One strong key and value, everything else silent: what the last query reads of it is the decay to the power of the distance."""
    from pico_engine.ops import kernels
    H, D, Dv, n, decay = 2, 32, 16, 512, [0.998, 0.99]
    qk = torch.zeros(n, 2, H, D)
    qk[n - 1, 0, :, 5] = 2.0
    qk[far, 1, :, 5] = 3.0
    proj = torch.zeros(n, H * Dv).to(torch.bfloat16)
    proj[far] = 4.0
    state = torch.zeros(2, H * D * Dv).cuda()
    one = lambda v: torch.tensor(v, dtype=torch.int32).cuda()
    o = kernels.linear_attention(proj.cuda(), 0, H * D, 0, H, D, Dv, state, 0, one([0, n]), one([n]), one([0]), chunked,
                                 head_decay=torch.tensor(decay).cuda(), qk=qk.reshape(n, 2 * H * D).cuda()).cpu().view(n, H, Dv)
    for h in range(H):
        want = 24.0 * decay[h] ** (n - 1 - far)
        assert (o[n - 1, h] - want).abs().max() < 1e-4 * 24.0


# ------------------------------------------------------------------ the window and the kept first tokens

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 32, 16), (8, 1, 64, 64), (2, 1, 128, 128), (3, 3, 24, 40)])
@pytest.mark.parametrize("window,keep", [(33, 3), (70, 100), (2, 1), (130, 64), (64, 65), (1, 5)])
def test_window_and_kept_token_edges_in_prompt_portions_and_decoding(dtype, H, G, D, Dv, window, keep):
    """One key at a time is made to dominate every query: those that see it give its value, those that do not give next to nothing of it.
    The key stands at a sequence's first places, at the last kept token and the one behind it, and beside page borders."""
    from pico_engine.ops import kernels
    dt = DTYPES[dtype]
    for key_at in sorted({0, keep - 1, keep, 63, 64, 128}):
        n = key_at + window + 70
        g = torch.Generator().manual_seed(key_at)
        q, k, v = (0.01 * torch.randn(n, h, d, generator=g) for h, d in ((H, D), (G, D), (G, Dv)))
        q[:, :, D - 1] = 6.0
        k[key_at, :, D - 1] = 6.0                                            # a score of 36 for every query
        v[key_at] = 10.0
        kp, table = cached(n, G, D, dt)
        vp, _ = cached(n, G, Dv, dt)
        for pool, src in ((kp, k), (vp, v)):
            pages = table.shape[1]
            padded = torch.zeros(pages * 64, G, src.shape[2])
            padded[:n] = src
            pool[2:] = padded.view(pages, 64, G, -1).permute(0, 2, 1, 3).to(dt).cuda()
        seen = plain.visible(n, window, keep)[:, key_at]
        edges = sorted({key_at, key_at + window - 1, key_at + window, key_at + window + 1, n - 1})
        for spans in ([(0, n)], [(0, key_at + 2), (key_at + 2, key_at + 4), (key_at + 4, n)], [(p, p + 1) for p in edges]):
            for a, b in spans:
                ctx = SimpleNamespace(one_token_each=(b - a == 1), scratch={}, lens=[b - a], starts=[a], max_context=b, dtype=dt)
                o = kernels.attention_headmix(q[a:b].reshape(b - a, H * D).to(dt).cuda().contiguous(), H * D, H, G, D, Dv, kp, vp, table, table.shape[1],
                                              torch.arange(a, b, dtype=torch.int32).cuda(), torch.zeros(b - a, dtype=torch.int32).cuda(), window, 1.0,
                                              None, None, ctx, keep_first=keep).float().cpu().view(b - a, H, Dv)
                s = seen[a:b]
                assert (o[s] - 10.0).abs().max() < 0.05 if s.any() else True, (key_at, a, b)
                assert o[~s].abs().max() < 0.1 if (~s).any() else True, (key_at, a, b)


# ------------------------------------------------------------------ relu gate

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("I", [64, 27, 4864])
def test_relu_gate(dtype, I):
    from pico_engine.ops import kernels
    dt = DTYPES[dtype]
    gu = torch.randn(9, 2 * I, generator=torch.Generator().manual_seed(I)).to(dt)
    want = torch.clamp(gu[:, :I].double(), min=0) * gu[:, I:].double()
    got = kernels.gated_act(gu.cuda(), "relu").double().cpu()
    assert (got - want).abs().max() < (4e-2 if dtype == "bfloat16" else 1e-6)
    assert not got[gu[:, :I].double() < 0].any()


@pytest.mark.parametrize("activation", ["relu", "silu"])
@pytest.mark.parametrize("M,K,I", [(1, 64, 24), (3, 72, 100), (8, 896, 4864), (9, 200, 72), (16, 1024, 512)])
def test_gate_up_and_activation_of_a_decode_step_in_one_kernel(activation, M, K, I):
    from pico_engine.ops import kernels
    from pico_engine.ops.linear import gate_up_act
    g = torch.Generator().manual_seed(M * 10 + I)
    h, w = torch.randn(M, K, generator=g).bfloat16(), (torch.randn(2 * I, K, generator=g) * K ** -0.5).bfloat16()
    gate, up = h.double() @ w[:I].double().T, h.double() @ w[I:].double().T
    want = (torch.clamp(gate, min=0) if activation == "relu" else gate * plain.sigmoid(gate)) * up
    fused = I % 8 == 0
    if fused:
        got = kernels.gate_up_act(h.cuda(), w.cuda(), activation).double().cpu()
        assert (got - want).abs().max() < 3e-2 * max(1.0, float(want.abs().max()))
        if activation == "relu":
            assert not got[gate < -0.05].any()
    got = gate_up_act(h.cuda(), w.cuda(), activation).double().cpu()
    assert got.shape == (M, I) and (got - want).abs().max() < 3e-2 * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("orientation", ["rows", "swapped", "pairs"])
@pytest.mark.parametrize("M,K,I", [(17, 128, 64), (100, 896, 304), (300, 200, 1000)])
def test_relu_gate_in_the_epilogue_of_the_tcgen05_product(orientation, M, K, I):
    from pico_engine.ops import kernels
    g = torch.Generator().manual_seed(M + I)
    h, w = torch.randn(M, K, generator=g).bfloat16(), (torch.randn(2 * I, K, generator=g) * K ** -0.5).bfloat16()
    gate, up = h.double() @ w[:I].double().T, h.double() @ w[I:].double().T
    got = kernels.gemm_tcgen05(h.cuda(), w.cuda(), swiglu="relu", orientation=orientation).double().cpu()
    want = torch.clamp(gate, min=0) * up
    assert (got - want).abs().max() < 3e-2 * max(1.0, float(want.abs().max()))
    kernels.check_status(torch.device("cuda", 0))
