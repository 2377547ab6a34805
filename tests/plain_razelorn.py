"""A plain, slow implementation of the Razelorn decoder: whole sequences, no cache, no batching, one function per
mechanism, written out from the design's equations.  It shares no code with the library and is the oracle of the
GPU tests.

Notation.  A sequence has tokens at positions p = 0 .. n-1; ``x`` is the residual stream [n, width].  ``cfg`` is the
parsed config.json, ``w`` maps tensor names to tensors; matrices are [out, in] and applied as W x.  Everything runs
in the dtype of the weights handed in (the tests use float64).
"""
from __future__ import annotations

import math

import torch

ROUTER_GAPS = None      # a list here receives, for every router run, each token's distance between the last chosen and the first other choice score


# ------------------------------------------------------------------ small pieces

def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, bias, eps):
    """(x - mean) / sqrt(var + eps) * weight + bias over the last axis, var the mean of the squared deviations."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def lin(w, h):
    return h @ w.T


# ------------------------------------------------------------------ rotation

def frequencies(dims, base, scaling=None):
    """f_i = base^(-2i/dims), i < dims/2.  With ``scaling`` (factor, low, high, original) the wavelength l = 2 pi / f decides:
    below original / high the frequency stays, above original / low it is divided by the factor, in between the two are mixed by
    s = (original / l - low) / (high - low)."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            factor, low, high, original = (scaling[k] for k in ("factor", "low", "high", "original"))
            wave = 2 * math.pi / f
            if wave > original / low:
                f = f / factor
            elif wave >= original / high:
                s = (original / wave - low) / (high - low)
                f = (1 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate_half(u, dims, freqs):
    """u [n, ..., D]: entry i < dims/2 pairs with entry i + dims/2; the pair (a, b) of the token at position p becomes
    (a cos - b sin, b cos + a sin) with the angle p * freqs[i].  Entries from ``dims`` on stay."""
    out = u.clone()
    pos = torch.arange(u.shape[0], dtype=u.dtype)
    half = dims // 2
    for i in range(half):
        shape = (-1,) + (1,) * (u.dim() - 2)
        c, s = torch.cos(pos * freqs[i]).view(shape), torch.sin(pos * freqs[i]).view(shape)
        a, b = u[..., i], u[..., i + half]
        out[..., i] = a * c - b * s
        out[..., i + half] = b * c + a * s
    return out


# ------------------------------------------------------------------ attention

def window_mask(n, size=None):
    """[n, n] bool: i sees j iff 0 <= i - j (< size where there is one)."""
    d = torch.arange(n).view(-1, 1) - torch.arange(n).view(1, -1)
    return (d >= 0) if size is None else (d >= 0) & (d < size)


def softmax_rows(s, seen):
    s = torch.where(seen, s, torch.full_like(s, -math.inf))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def mixing_number(w, p, diff):
    """lambda: one number a layer."""
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def difference_of_maps(a1, a2, lam, diff, eps):
    """a1, a2 [n, vdim], the outputs of a head's two maps."""
    return rms_unit(a1 - lam * a2, eps) * (1 - diff)


def query_key_heads(h, m, w, p, eps):
    """(q [n, H, 2, dim], k [n, G, 2, dim]) normed and rotated."""
    n, D = h.shape[0], m["dim"]
    q = lin(w[p + "q"], h).view(n, m["heads"], 2, D)
    k = lin(w[p + "k"], h).view(n, m["kv_heads"], 2, D)
    q, k = rms_unit(q, eps) * w[p + "q.norm"], rms_unit(k, eps) * w[p + "k.norm"]
    rot = m.get("rot")
    if rot is not None and rot["dims"]:
        f = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q, k = rotate_half(q, rot["dims"], f), rotate_half(k, rot["dims"], f)
    return q, k


def differential_heads(q, k, v, scale, size, lam, diff, eps):
    """[n, H, vdim] of q [n, H, 2, dim], k [n, G, 2, dim], v [n, G, vdim]."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    seen = window_mask(n, size)
    out = []
    for h in range(H):
        g = h // (H // G)
        a1, a2 = (softmax_rows((q[:, h, t] @ k[:, g, t].T) * scale, seen) @ v[:, g] for t in (0, 1))
        out.append(difference_of_maps(a1, a2, lam, diff, eps))
    return torch.stack(out, dim=1)


def attention_mixer(h, m, w, p, eps):
    n = h.shape[0]
    q, k = query_key_heads(h, m, w, p, eps)
    v = lin(w[p + "v"], h).view(n, m["kv_heads"], m["vdim"])
    size = (m.get("mask") or {}).get("size")
    o = differential_heads(q, k, v, m["scale"], size, mixing_number(w, p, m["diff"]), m["diff"], eps)
    return lin(w[p + "o"], o.reshape(n, -1))


# ------------------------------------------------------------------ feed-forwards

def dense_ff(h, w, p):
    return lin(w[p + "down"], torch.clamp(lin(w[p + "up"], h), min=0) ** 2)


def expert(h, w, p):
    z = lin(w[p + "gate"], h)
    return lin(w[p + "down"], z * sigmoid(z) * lin(w[p + "up"], h))


def route(h, mlp, w, p):
    """For every token the list of (expert, weight): scores are the softmax over all outputs of the router, the choice reads
    score + correction, the weight is the score."""
    z = lin(w[p + "router"], h)
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    c, top = s + w[p + "correction"], mlp["router"]["top"]
    out, gaps = [], []
    for t in range(h.shape[0]):
        ranked = torch.argsort(c[t], descending=True, stable=True).tolist()
        gaps.append(float(c[t, ranked[top - 1]] - c[t, ranked[top]]) if top < len(ranked) else math.inf)
        out.append([(j, s[t, j]) for j in ranked[:top]])
    if ROUTER_GAPS is not None:
        ROUTER_GAPS.append(torch.tensor(gaps))
    return out


def moe_ff(h, mlp, w, p):
    r = mlp["router"]
    rows = []
    for t, chosen in enumerate(route(h, mlp, w, p)):
        y = torch.zeros_like(h[t])
        for e, weight in chosen:
            y = y + weight * (h[t] if e >= r["experts"] else expert(h[t], w, f"{p}e{e}."))
        if mlp.get("shared") is not None:
            y = y + sigmoid(lin(w[p + "shared.sg"], h[t])) * expert(h[t], w, p + "shared.")
        rows.append(y)
    return torch.stack(rows)


# ------------------------------------------------------------------ the model

def weights_layer(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def hidden_states(cfg, w, tokens, keep_layers=False):
    """The residual stream after the last layer [n, width] (``keep_layers``: the list of streams after every layer too)."""
    eps = cfg["norm"]["eps"]
    x = torch.stack([w["embed"][t] for t in tokens]) * cfg["embedding"]["scale"]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{weights_layer(cfg, i)}.", layer["mixer"], layer.get("mlp")
        if layer["type"] != "attention":
            raise ValueError(f"unknown layer type {layer['type']!r}")
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        y = attention_mixer(h, m, w, p + "mix.", eps)
        if mlp is not None:
            y = y + (dense_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(h, mlp, w, p + "mlp."))
        x = x + y
        after.append(x)
    return (x, after) if keep_layers else x


def logits(cfg, w, tokens):
    """[n, vocab]."""
    x = hidden_states(cfg, w, tokens)
    return lin(w["head"], layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"]))


def greedy(cfg, w, prompt, n_new):
    tokens, out = list(prompt), []
    for _ in range(n_new):
        t = int(torch.argmax(logits(cfg, w, tokens)[-1]))
        out.append(t)
        tokens.append(t)
    return out
