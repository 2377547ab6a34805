"""Small Razelorn configurations and random weights for the tests, written out independently of the library.

The configurations differ from one another in every size and option: 1, 3, 4 and 17 query heads a key/value head; values smaller than,
equal to and larger than keys, at sizes of every attention kernel; rotation of all, some and none of a head's entries, by bands of
wavelengths that keep, mix and divide, or unscaled; windows of 1, 2, 33, 70, 130 tokens, exactly a page, and none; lambda bases 0, below
zero and above; mixtures with and without identity experts and shared expert, top 1, top = all outputs and in between, hidden sizes
that are multiples of nothing; dense and absent feed-forwards; layers that use the tensors of an earlier one, of a later one and of one
that itself uses another's; embedding scales including 1.
"""
from __future__ import annotations

import torch


def attention(heads, kv_heads, dim, vdim, scale, diff, window=None, rot=None, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = {"base": rot[1], "dims": rot[0]}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=None, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if identity is not None:
        m["router"]["identity"] = identity
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp, weights_of=None):
    d = {"type": "attention", "mixer": mixer, "mlp": mlp}
    if weights_of is not None:
        d["weights_of"] = weights_of
    return d


def config(vocab, width, eps, scale, layers):
    return {"architecture": "Razelorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


A1 = attention(6, 2, 32, 24, 0.22, 0.4, 70, (16, 1000.0), (4.0, 1.0, 4.0, 64))
M1 = moe(6, 3, 24, identity=3, shared=40)
A3 = attention(3, 1, 12, 10, 0.35, -0.1, 33, (10, 100.0), (8.0, 0.5, 3.0, 40))
A4 = attention(4, 1, 64, 128, 0.15, 0.7, 130, (48, 40000.0), (8.0, 1.0, 2.0, 256))
A5 = attention(17, 1, 80, 136, 0.12, 0.25, 64)

CONFIGS = {
    # a page and a bit of window; bands inside the entries; a chain of layers on one mixture's tensors; a layer without feed-forward
    "R1": config(300, 80, 1e-5, 3.0, [layer(A1, M1), layer(attention(2, 2, 48, 80, 0.15, 0.2, 2, (48, 300.0)), None), layer(A1, M1, 0), layer(A1, M1, 2)]),
    # no window, no bands, one query head a key/value head, no identity and no shared expert, top = every expert; diff = 0, scale 1
    "R2": config(128, 48, 1e-3, 1.0, [layer(attention(4, 4, 16, 16, 0.3, 0.0, None, (16, 50.0)), moe(2, 2, 16)),
                                      layer(attention(3, 3, 32, 16, 0.2, 0.5, None, (8, 50.0), (2.0, 1.0, 8.0, 30)), moe(3, 2, 16, shared=24))]),
    # sizes that are multiples of nothing (the kernels for any size), a width that is no multiple of 4, windows of 33 and 1; identity
    # experts without a shared one; the first layer uses a later layer's tensors
    "R3": config(90, 50, 2e-6, 0.5, [layer(A3, dense(37), 2), layer(attention(2, 1, 20, 6, 0.3, 0.3, 1, (4, 20.0)), moe(3, 1, 20, identity=2)),
                                     layer(A3, dense(37)), layer(attention(2, 2, 24, 12, 0.3, 0.9, None, (0, 100.0)), moe(4, 6, 13, identity=2, shared=11))]),
    # the largest sizes of the tcgen05 prompt kernel, a window above two pages; the same tensors three times
    "R4": config(200, 128, 1e-5, 8.0, [layer(A4, moe(8, 2, 32, identity=1, shared=48)), layer(A4, dense(160)), layer(A4, dense(160), 1), layer(A4, dense(160), 1)]),
    # the mma.sync prompt kernel's sizes, 17 query heads on one key/value head (two row tiles), a window of exactly a page, no rotation
    "R5": config(160, 96, 1e-4, 2.0, [layer(A5, dense(64)), layer(attention(8, 2, 96, 64, 0.11, 0.3, None, (96, 5000.0)), moe(4, 2, 32, identity=0, shared=32))]),
}


def owner(cfg, i):
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def tensor_shapes(cfg: dict) -> dict:
    W, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, W), "final.norm": (W,), "final.norm.b": (W,), "head": (V, W)}
    for i, l in enumerate(cfg["layers"]):
        if owner(cfg, i) != i:
            continue
        p, m, mlp = f"l{i}.mix.", l["mixer"], l["mlp"]
        H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        shapes.update({f"l{i}.norm1": (W,), f"l{i}.norm1.b": (W,), p + "q": (2 * H * D, W), p + "k": (2 * G * D, W), p + "v": (G * Dv, W),
                       p + "o": (W, H * Dv)})
        shapes.update({p + n: (D,) for n in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2")})
        q = f"l{i}.mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            shapes.update({q + "up": (mlp["ff"], W), q + "down": (W, mlp["ff"])})
            continue
        E, I, F = mlp["router"]["experts"], mlp["router"].get("identity", 0), mlp["expert"]["ff"]
        shapes.update({q + "router": (E + I, W), q + "correction": (E + I,)})
        for e in range(E):
            shapes.update({f"{q}e{e}.gate": (F, W), f"{q}e{e}.up": (F, W), f"{q}e{e}.down": (W, F)})
        if "shared" in mlp:
            S = mlp["shared"]["ff"]
            shapes.update({q + "shared.gate": (S, W), q + "shared.up": (S, W), q + "shared.down": (W, S), q + "shared.sg": (1, W)})
    return shapes


def make_weights(cfg: dict, seed: int, steady_routing: bool = False) -> dict:
    """Random weights rounded to bfloat16 values (kept in float32 here).  ``steady_routing``: corrections more than a score apart, so that
    rounding cannot turn a choice (for runs in bfloat16); otherwise corrections of the scores' own spread, so that the choice varies from
    token to token."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm"):
            t = 1.0 + 0.1 * torch.randn(shape, generator=g)
        elif last == "b":
            t = 0.2 * torch.randn(shape, generator=g)
        elif last in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.3 * torch.randn(shape, generator=g)
        elif last == "router":
            t = torch.randn(shape, generator=g) * 1.5 * shape[1] ** -0.5
        elif last == "correction":
            t = torch.randperm(shape[0], generator=g).float() * 1.25 if steady_routing else 0.15 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g) * 0.7 / max(cfg["embedding"]["scale"], 1.0) ** 0.5
        else:
            t = torch.randn(shape, generator=g) * shape[1] ** -0.5
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out


def requests_for(cfg: dict, lengths, seed: int = 7) -> dict:
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}


_cache = {}
CLOSE_CALL = 0.02


def plain_logits(cfg: dict, weights: dict, requests: dict, close_calls: set | None = None) -> dict:
    """{(request, position): logits row} of the plain implementation in float64 (kept: the tests ask for the same requests in several ways
    of cutting).  ``close_calls`` receives the places at which some router of the plain run chose its last expert by less than
    CLOSE_CALL."""
    import plain_razelorn as plain
    out, w64 = {}, None
    for rid, toks in requests.items():
        key = (id(weights), tuple(toks))
        if key not in _cache:
            if w64 is None:
                w64 = {n: t.double() for n, t in weights.items()}
            plain.ROUTER_GAPS = []
            with torch.no_grad():
                logits = plain.logits(cfg, w64, toks).float().numpy()
            gaps, plain.ROUTER_GAPS = plain.ROUTER_GAPS, None
            close = torch.stack(gaps).min(0).values < CLOSE_CALL if gaps else torch.zeros(len(toks), dtype=torch.bool)
            _cache[key] = (logits, close.tolist())
        logits, close = _cache[key]
        for p in range(len(toks)):
            out[(rid, p)] = logits[p]
            if close_calls is not None and close[p]:
                close_calls.add((rid, p))
    return out
