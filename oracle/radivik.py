"""Plain CPU restatement of the Radivik decoder, one function per mechanism, in numpy (float64 by default).

Test infrastructure: only tests import it, and it shares no code with the product path.  Everything is written for a
whole sequence at once, with no cache: the product's cache, portions and batches are what it checks.

Weights are a dict of arrays named as in a checkpoint ('embed', 'l0.mix.q', 'l0.mlp.e3.gate', 'final.norm', 'head').
"""
from __future__ import annotations

import math

import numpy as np


def rms_norm(x, eps, weight=None):
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def rotary_frequencies(rot):
    """(frequencies [dims / 2], multiplier of cos and sin).  With scaling, slow components are stretched by `factor`,
    fast ones kept, and a linear ramp over the component index joins the two."""
    dims, base = rot["dims"], float(rot["base"])
    i = np.arange(dims // 2, dtype=np.float64)
    f = base ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def index_of(turns):  # component whose wave makes `turns` turns within the original context
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(index_of(sc["fast"])), 0), min(math.ceil(index_of(sc["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, heads, dim]: the first rot.dims channels turn in pairs (i, i + dims / 2), the rest pass."""
    f, mult = rotary_frequencies(rot)
    half = rot["dims"] // 2
    a = np.asarray(positions, np.float64)[:, None] * f
    c, s = (np.cos(a) * mult)[:, None, :], (np.sin(a) * mult)[:, None, :]
    u, v = x[..., :half], x[..., half : 2 * half]
    out = np.array(x, np.float64)
    out[..., :half] = u * c - v * s
    out[..., half : 2 * half] = v * c + u * s
    return out


def causal_attention(q, k, v, scale, first=0):
    """q [T, H, dim] at positions first.., k [S, G, dim], v [S, G, vdim] from position 0.  Query i sees keys j <= first + i."""
    T, H, _ = q.shape
    S, G, vdim = v.shape
    out = np.zeros((T, H, vdim))
    visible = np.arange(S)[None, :] <= first + np.arange(T)[:, None]
    for h in range(H):
        g = h // (H // G)
        s = np.where(visible, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        p = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[:, g]
    return out


def attention_keys_values(h, w, p, mx, positions, eps):
    """Keys (rotated, then of unit root mean square) and values of a layer that has projections of its own."""
    T = h.shape[0]
    k = (h @ w[p + "k"].T).reshape(T, mx["kv_heads"], mx["dim"])
    if mx.get("rot"):
        k = rotate(k, positions, mx["rot"])
    return rms_norm(k, eps), (h @ w[p + "v"].T).reshape(T, mx["kv_heads"], mx["vdim"])


def attention(h, w, p, mx, positions, eps, kv):
    T = h.shape[0]
    q = (h @ w[p + "q"].T).reshape(T, mx["heads"], mx["dim"])
    if mx.get("rot"):
        q = rotate(q, positions, mx["rot"])
    out = causal_attention(rms_norm(q, eps), kv[0], kv[1], mx["scale"])
    return out.reshape(T, -1) @ w[p + "o"].T


def expert(h, w, p, limit):
    g = np.minimum(h @ w[p + "gate"].T, limit)
    u = np.clip(h @ w[p + "up"].T, -limit, limit)
    return (g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)) @ w[p + "down"].T


def route(h, router, top):
    """(chosen experts [T, top], their scores)."""
    s = 1.0 / (1.0 + np.exp(-(h @ router.T)))
    ids = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return ids, np.take_along_axis(s, ids, axis=1)


def margin(h, router, top):
    """How far apart the last chosen and the first unchosen score of every token are (infinite without the latter)."""
    s = np.sort(1.0 / (1.0 + np.exp(-(h @ router.T))), axis=1)
    return s[:, -top] - s[:, -top - 1] if top < s.shape[1] else np.full(len(h), np.inf)


def mixture(h, w, p, mlp, margins=None):
    ids, s = route(h, w[p + "router"], mlp["router"]["top"])
    if margins is not None:
        margins.append(margin(h, w[p + "router"], mlp["router"]["top"]))
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, slot = np.nonzero(ids == e)
        if len(t):
            out[t] += expert(h[t] * s[t, slot][:, None], w, f"{p}e{e}.", mlp["expert"]["limit"])
    return out


def forward(cfg, w, tokens, dtype=np.float64, margins=None):
    """(logits [T, vocab], residual stream after every layer [layers, T, width]).  `margins`: receives every router's."""
    w = {k: np.asarray(v, dtype) for k, v in w.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    positions = np.arange(len(tokens))
    x = w["embed"][np.asarray(tokens)]
    kvs, after = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        src = mx.get("kv_from")
        if src is None:
            kvs[i] = attention_keys_values(x, w, p + "mix.", mx, positions, eps)
        kv = kvs[i if src is None else src]
        x = rms_norm(alpha * x + attention(x, w, p + "mix.", mx, positions, eps, kv), eps, w[p + "norm1"])
        if layer.get("mlp"):
            x = rms_norm(alpha * x + mixture(x, w, p + "mlp.", layer["mlp"], margins), eps, w[p + "norm2"])
        after.append(x)
    return rms_norm(x, eps, w["final.norm"]) @ w["head"].T, np.stack(after)
