"""A plain, slow implementation of the Lefilorn decoder: whole sequences, no cache, no batching, one function per
mechanism, written out from the design's equations.  It shares no code with the library and is the oracle of the
GPU tests.

Notation.  A sequence has tokens at positions p = 0 .. n-1; the residual is a list of ``streams`` matrices [n, width].
``cfg`` is the parsed config.json, ``w`` maps tensor names to tensors; matrices are [out, in] and applied as W x.
Everything runs in the dtype of the weights handed in (the tests use float64).
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------ small pieces

def unit_rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def lin(w, h):
    return h @ w.T


# ------------------------------------------------------------------ rotations

def frequency(i, dims, base):
    return base ** (-2.0 * i / dims)


def turned(u, v, p, f):
    """The pair (u, v) [n, heads] of the tokens at positions ``p`` [n], turned by p * f."""
    a = (p * f)[:, None]
    c, s = torch.cos(a), torch.sin(a)
    return u * c - v * s, v * c + u * s


def rotate_neighbours(x, dims, base, first=0):
    """x [n, heads, D]: entries 2i and 2i+1 of the first ``dims`` form a pair; the rest of a head stays."""
    out = x.clone()
    p = torch.arange(first, first + x.shape[0], dtype=x.dtype)
    for i in range(dims // 2):
        out[..., 2 * i], out[..., 2 * i + 1] = turned(x[..., 2 * i], x[..., 2 * i + 1], p, frequency(i, dims, base))
    return out


def rotate_halves(x, dims, base, first=0):
    """x [n, heads, D]: entries i and i + dims/2 of the first ``dims`` form a pair; the rest of a head stays."""
    out = x.clone()
    p = torch.arange(first, first + x.shape[0], dtype=x.dtype)
    half = dims // 2
    for i in range(half):
        out[..., i], out[..., i + half] = turned(x[..., i], x[..., i + half], p, frequency(i, dims, base))
    return out


# ------------------------------------------------------------------ softmax attention with a window and kept first tokens

def visible(n, size=None, keep_first=0):
    """[n, n] bool: i sees j iff j <= i and (i - j < size or j < keep_first); without a size every j <= i."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    seen = j <= i
    if size is not None:
        seen = seen & ((i - j < size) | (j < keep_first))
    return seen


def attention(q, k, v, scale, seen):
    """q [n, H, D], k [n, G, D], v [n, G, Dv] -> [n, H, Dv]; query head h reads key/value head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        c = h // (H // G)
        s = (q[:, h] @ k[:, c].T) * scale
        s = s.masked_fill(~seen, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out.append((e / e.sum(-1, keepdim=True)) @ v[:, c])
    return torch.stack(out, dim=1)


def attention_branch(h, w, p, m, eps):
    """The left mixer: biased projections, q and k normed over all their rows at once, rotation of neighbours, the
    window with kept first tokens, a sigmoid gate on the concatenated heads."""
    n = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm(lin(w[p + "q"], h) + w[p + "q.b"], w[p + "q.norm"], eps).view(n, H, D)
    k = rms_norm(lin(w[p + "k"], h) + w[p + "k.b"], w[p + "k.norm"], eps).view(n, G, D)
    v = (lin(w[p + "v"], h) + w[p + "v.b"]).view(n, G, Dv)
    q, k = rotate_neighbours(q, m["rot"]["dims"], m["rot"]["base"]), rotate_neighbours(k, m["rot"]["dims"], m["rot"]["base"])
    mask = m.get("mask") or {}
    o = attention(q, k, v, m["scale"], visible(n, mask.get("size"), mask.get("keep_first", 0))).reshape(n, H * Dv)
    return lin(w[p + "o"], o * sigmoid(lin(w[p + "g"], h)))


# ------------------------------------------------------------------ retention

def retention(q, k, v, decay):
    """S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head, S = 0 before the first token; q, k [n, H, D], v [n, H, Dv]."""
    n, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    a = torch.tensor(decay, dtype=q.dtype).view(H, 1, 1)
    out = []
    for t in range(n):
        S = a * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def retention_branch(h, w, p, m, eps):
    """The right mixer: rotation of halves, keys scaled by dim^(-1/2), every head's output divided by its root mean
    square, a silu gate on the concatenated heads."""
    n = h.shape[0]
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    q = rotate_halves(lin(w[p + "q"], h).view(n, H, D), m["rot"]["dims"], m["rot"]["base"])
    k = rotate_halves(lin(w[p + "k"], h).view(n, H, D), m["rot"]["dims"], m["rot"]["base"]) * D ** -0.5
    v = lin(w[p + "v"], h).view(n, H, Dv)
    o = unit_rms(retention(q, k, v, m["decay"]), eps).reshape(n, H * Dv)
    g = lin(w[p + "g"], h)
    return lin(w[p + "o"], o * (g * sigmoid(g)))


def side_by_side(h, w, p, m, eps):
    return (m["left_scale"] * attention_branch(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * retention_branch(h, w, p + "right.", m["right"], eps))


# ------------------------------------------------------------------ feed-forward

def relu_gated(h, w, p):
    return lin(w[p + "down"], torch.clamp(lin(w[p + "gate"], h), min=0.0) * lin(w[p + "up"], h))


# ------------------------------------------------------------------ streams

def streams_in(xs, weights):
    """What a sublayer reads: the weighted sum of the streams."""
    return sum(weights[s] * x for s, x in enumerate(xs))


def streams_out(xs, y, mix, out):
    """Every stream from all the old ones (mix[from, to]) and its share of the sublayer's output."""
    return [sum(mix[s, t] * x for s, x in enumerate(xs)) + out[t] * y for t in range(len(xs))]


def run_sublayer(xs, w, p, number, norm, eps, fn):
    """One sublayer around the streams; without streams in the design (``xs`` of one entry and no such tensors): x + fn(norm(x))."""
    q = f"{p}hc{number}."
    if q + "in" not in w:
        (x,) = xs
        return [x + fn(rms_norm(x, w[p + norm], eps))]
    y = fn(rms_norm(streams_in(xs, w[q + "in"]), w[p + norm], eps))
    return streams_out(xs, y, w[q + "mix"], w[q + "out"])


# ------------------------------------------------------------------ the model

def layer_runs(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def hidden(tokens, w, cfg, trace=None):
    """The sum of the streams after the last layer; ``trace`` (a list) receives that sum after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * (cfg.get("embedding") or {}).get("scale", 1.0)
    xs = [x0] * (cfg.get("streams") or 1)
    for i in layer_runs(cfg):
        p, layer = f"l{i}.", cfg["layers"][i]
        xs = run_sublayer(xs, w, p, 1, "norm1", eps, lambda h: side_by_side(h, w, p + "mix.", layer["mixer"], eps))
        if layer.get("mlp"):
            xs = run_sublayer(xs, w, p, 2, "norm2", eps, lambda h: relu_gated(h, w, p + "mlp."))
        if trace is not None:
            trace.append(sum(xs))
    return sum(xs)


def logits(tokens, w, cfg):
    """[n, vocab] for one sequence."""
    return lin(w["head"], rms_norm(hidden(tokens, w, cfg), w["final.norm"], cfg["norm"]["eps"]))


def generate(tokens, w, cfg, n_new):
    """Greedy continuation: recomputes the whole sequence for every new token."""
    tokens = list(tokens)
    for _ in range(n_new):
        tokens.append(int(torch.argmax(logits(tokens, w, cfg)[-1])))
    return tokens
