"""Small Lefilorn configurations and random weights for the tests, written out independently of the library.

The configurations differ from one another in every size and option: 1, 2, 3, 5 and 9 streams and none at all; loops that start at
the first layer, run once, end with the last layer, or are absent; 1, 2, 3 and 8 query heads a key/value head; values smaller than,
equal to and larger than keys; all, some and none of a head's entries rotated, on either side; windows of 1 and 2 tokens, below a
cache page, just above a page, above two pages and none, with no kept first tokens, one, a few, exactly a page, and more than the
window is long; linear attention with 1 to 4 heads, keys from 8 to 136 entries, decays of 1, 0 and in between; layers without a
feed-forward; branch factors of either sign; embedding scales including 1; norm constants from 2e-6 to 1e-2.  Weights have the scale
1/sqrt(inputs) so that activations keep their size and scores spread.
"""
from __future__ import annotations

import torch


def left(heads, kv_heads, dim, vdim, scale, rot, mask=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": dict(zip(("dims", "base"), rot))}
    if mask is not None:
        m["mask"] = dict(zip(("size", "keep_first"), mask))
    return m


def right(dim, vdim, decay, rot):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay), "rot": dict(zip(("dims", "base"), rot))}


def layer(a, b, scales, ff):
    return {"type": "parallel", "mixer": {"left": a, "right": b, "left_scale": scales[0], "right_scale": scales[1]},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, eps, scale, streams, layers, loop=None):
    d = {"architecture": "Lefilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if streams is not None:
        d["streams"] = streams
    if loop is not None:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


CONFIGS = {
    # two streams; the loop starts at the first layer and runs three times; half of a head rotated left, a part right; a window
    # below a page with three kept tokens; values smaller than keys left, larger right; a last layer without feed-forward
    "L1": config(300, 72, 5e-2, 3.0, 2, [
        layer(left(4, 2, 32, 16, 0.3, (16, 10000.0), (33, 3)), right(16, 24, [0.9, 0.5, 1.0], (8, 500.0)), (0.5, 0.6), 100),
        layer(left(4, 2, 32, 16, 0.3, (16, 10000.0), (33, 3)), right(16, 24, [0.9, 0.5, 1.0], (8, 500.0)), (0.5, 0.6), 64),
        layer(left(2, 2, 16, 16, 0.6, (16, 300.0), (65, 1)), right(40, 8, [0.97], (40, 10000.0)), (-0.6, 0.4), None)], loop=(0, 2, 3)),
    # one stream (its mix is a number); no loop; values larger than keys; no window; nothing rotated right, a pair left; decay 0
    "L2": config(128, 48, 3e-2, 1.0, 1, [
        layer(left(3, 1, 16, 40, 0.7, (2, 50.0)), right(32, 48, [1.0, 0.0], (0, 7.0)), (1.0, 0.5), 40),
        layer(left(6, 3, 24, 24, 0.5, (0, 50.0), (70,)), right(8, 8, [0.999, 0.6, 0.3, 0.9], (8, 100.0)), (0.5, 1.0), 56)]),
    # head size 64 (the tensor-memory prompt kernel and the cluster kernel), eight query heads on one key/value head; more kept tokens
    # than the window is long; five streams; a loop of one pass in the middle
    "L3": config(200, 128, 1e-2, 8.0, 5, [
        layer(left(8, 1, 64, 64, 0.3, (64, 40000.0), (70, 100)), right(64, 64, [0.99, 0.9], (48, 40000.0)), (0.9, 0.8), 160),
        layer(left(2, 2, 64, 64, 0.25, (32, 1000.0), (130, 64)), right(32, 16, [0.8, 0.998, 0.95], (32, 1000.0)), (0.4, 1.1), 96),
        layer(left(8, 1, 64, 64, 0.3, (64, 40000.0), (45,)), right(64, 64, [0.99, 0.9], (48, 40000.0)), (0.9, 0.8), 160)], loop=(1, 2, 1)),
    # sizes that are multiples of nothing, nine streams (more than the vector kernel takes), windows of two tokens and of one with kept
    # tokens; the loop ends with the last layer
    "L4": config(90, 50, 2e-2, 0.5, 9, [
        layer(left(3, 1, 24, 12, 0.3, (10, 100.0), (2, 1)), right(20, 12, [0.5, 0.9, 0.999], (6, 100.0)), (0.5, 0.3), 36),
        layer(left(5, 5, 10, 22, 0.4, (10, 20.0), (1, 5)), right(12, 30, [0.95], (12, 20.0)), (0.5, 0.4), 27)], loop=(1, 2, 2)),
    # no streams (one plain residual sum); head size 128 left, 136 right (more than 128 key channels); kept tokens beside a window of
    # more than two pages
    "L5": config(160, 96, 1e-2, 2.0, None, [
        layer(left(2, 1, 128, 128, 0.2, (96, 5000.0), (150, 7)), right(136, 40, [0.97, 0.7], (136, 5000.0)), (0.6, 0.7), 120),
        layer(left(4, 2, 48, 32, 0.35, (48, 5000.0), (64, 64)), right(24, 72, [0.9, 1.0], (12, 5000.0)), (1.0, 1.0), None)], loop=(0, 1, 2)),
    # three streams; everything once more at other sizes, the two factors equal, one layer that is no loop
    "L6": config(97, 64, 2e-6, 5.0, 3, [
        layer(left(4, 4, 32, 32, 0.5, (32, 200.0), (20, 2)), right(16, 16, [0.96, 0.8], (16, 900.0)), (0.5, 0.5), 88)]),
}


# Seeds of the weights the whole-model tests take: models in which rounding stays rounding.  (Dividing every head of the linear branch by
# its root mean square can blow up a head that is nearly zero, at a sequence's first tokens above all; the constants above bound that,
# and these draws have no such head in front of a long run of layers.)
SEEDS = {"L1": 124, "L2": 121, "L3": 122, "L4": 120, "L5": 124, "L6": 125}


def tensor_shapes(cfg: dict) -> dict:
    W, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        a, b = l["mixer"]["left"], l["mixer"]["right"]
        H, G, D, Dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        q = p + "mix.left."
        shapes.update({p + "norm1": (W,), q + "q": (H * D, W), q + "q.b": (H * D,), q + "k": (G * D, W), q + "k.b": (G * D,), q + "v": (G * Dv, W),
                       q + "v.b": (G * Dv,), q + "q.norm": (H * D,), q + "k.norm": (G * D,), q + "g": (H * Dv, W), q + "o": (W, H * Dv)})
        H, D, Dv = b["heads"], b["dim"], b["vdim"]
        q = p + "mix.right."
        shapes.update({q + "q": (H * D, W), q + "k": (H * D, W), q + "v": (H * Dv, W), q + "g": (H * Dv, W), q + "o": (W, H * Dv)})
        halves = ["hc1"]
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            shapes.update({p + "norm2": (W,), p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
            halves.append("hc2")
        S = cfg.get("streams")
        if S is not None:
            for hc in halves:
                shapes.update({f"{p}{hc}.in": (S,), f"{p}{hc}.out": (S,), f"{p}{hc}.mix": (S, S)})
    return shapes


def make_weights(cfg: dict, seed: int) -> dict:
    """Random weights rounded to bfloat16 values (kept in float32 here)."""
    g = torch.Generator().manual_seed(seed)
    S = cfg.get("streams") or 1
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        last = name.rsplit(".", 1)[-1]
        r = torch.randn(shape, generator=g)
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.15 * r
        elif last == "b":
            t = 0.4 * r
        elif last == "in":
            t = (1.0 + 0.6 * r) / S
        elif last == "out":
            t = 0.6 + 0.3 * r
        elif last == "mix":                                   # near the identity and not symmetric: [from, to] shows
            t = 0.8 * torch.eye(S) + 0.3 * S ** -0.5 * r
        elif name == "embed":
            t = r * 0.7 / max(cfg["embedding"]["scale"], 1.0) ** 0.5
        else:
            t = r * shape[1] ** -0.5
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out


def requests_for(cfg: dict, lengths, seed: int = 7) -> dict:
    g = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for i, n in enumerate(lengths)}


_cache = {}


def plain_logits(cfg: dict, weights: dict, requests: dict) -> dict:
    """{(request, position): logits row} of the plain implementation in float64 (kept: the tests ask for the same requests in
    several ways of cutting)."""
    import plain_lefilorn as plain
    out, w64 = {}, None
    for rid, toks in requests.items():
        key = (id(weights), tuple(toks))
        if key not in _cache:
            if w64 is None:
                w64 = {n: t.double() for n, t in weights.items()}
            with torch.no_grad():
                _cache[key] = plain.logits(toks, w64, cfg).float().numpy()
        for p in range(len(toks)):
            out[(rid, p)] = _cache[key][p]
    return out
