"""Plain CPU restatement of the Biranex decoder, one function per mechanism, in numpy (float64 by default).

Test infrastructure: only tests import it, and it shares no code with the product path.  Everything is written for a
whole sequence at once and token by token where a state is carried, with no cache: the product's cache, states, portions
and batches are what it checks.

Weights are a dict of arrays named as in a checkpoint ('embed', 'l0.mix.q', 'l1.mix.left.sink', 'final.norm').
"""
from __future__ import annotations

import numpy as np

UNIT_EPS = 1e-6


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rms_norm(x, eps, weight=None):
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + UNIT_EPS)


def rotate_interleaved(x, positions, rot):
    """x [T, heads, dim]: channels 2i and 2i + 1 below rot.dims turn together, the rest pass."""
    n = rot["dims"] // 2 if rot else 0
    out = np.array(x)
    for i in range(n):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"]) / float((rot.get("scaling") or {"factor": 1.0})["factor"])
        a = np.asarray(positions, np.float64) * f
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def window_attention(q, k, v, scale, window=0, sink=None):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim].  Query i sees keys i - window < j <= i (window 0: all j <= i);
    exp(sink[h]) joins the denominator of head h."""
    T, H, _ = q.shape
    G, vdim = v.shape[1:]
    out = np.zeros((T, H, vdim))
    for i in range(T):
        lo = max(0, i - window + 1) if window else 0
        for h in range(H):
            g = h // (H // G)
            s = (k[lo : i + 1, g] @ q[i, h]) * scale
            top = max(s.max(), -np.inf if sink is None else sink[h])
            p = np.exp(s - top)
            den = p.sum() + (0.0 if sink is None else np.exp(sink[h] - top))
            out[i, h] = (p / den) @ v[lo : i + 1, g]
    return out


def causal_conv(x, weight, bias=None):
    """x [T, channels], weight [channels, taps] (last column: the current token), zeros before the start."""
    taps = weight.shape[1]
    ext = np.concatenate([np.zeros((taps - 1, x.shape[1])), x])
    y = sum(ext[j : j + len(x)] * weight[:, j] for j in range(taps))
    return y if bias is None else y + bias


def state_space_scan(x, b, c, dt, a_log, d, state=None):
    """x [T, H, P], b and c [T, groups, N], dt [T, H] (positive): S <- exp(-exp(a_log) dt) S + dt b x^T, y = S^T c + d x."""
    T, H, P = x.shape
    G, N = b.shape[1:]
    S = np.zeros((H, N, P)) if state is None else state
    y = np.zeros((T, H, P))
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = np.exp(-np.exp(a_log[h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(b[t, g], x[t, h])
            y[t, h] = S[h].T @ c[t, g] + d[h] * x[t, h]
    return y


def gated_group_norm(y, z, groups, weight, eps):
    y = y * silu(z)
    T, n = y.shape
    return rms_norm(y.reshape(T, groups, n // groups), eps).reshape(T, n) * weight


def delta_scan(q, k, v, beta, decay, state=None):
    """q, k [T, Hk, dim], v [T, H, vdim], beta [T, H], decay [T, H, dim]:
    S <- decay * S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    T, H, P = v.shape
    Hk, D = k.shape[1:]
    S = np.zeros((H, D, P)) if state is None else state
    o = np.zeros((T, H, P))
    for t in range(T):
        for h in range(H):
            g = h // (H // Hk)
            S[h] *= decay[t, h][:, None]
            S[h] += np.outer(k[t, g], beta[t, h] * (v[t, h] - S[h].T @ k[t, g]))
            o[t, h] = S[h].T @ q[t, g]
    return o


def attention_half(h, w, p, m, eps):
    T = len(h)
    q = rms_norm(h @ w[p + "q"].T, eps, w[p + "q.norm"]).reshape(T, m["heads"], m["dim"])
    k = rms_norm(h @ w[p + "k"].T, eps, w[p + "k.norm"]).reshape(T, m["kv_heads"], m["dim"])
    v = (h @ w[p + "v"].T).reshape(T, m["kv_heads"], m["vdim"])
    q, k = rotate_interleaved(q, range(T), m["rot"]), rotate_interleaved(k, range(T), m["rot"])
    a = window_attention(q, k, v, m["scale"], m["mask"]["size"], w[p + "sink"])
    a = a * sigmoid(h @ w[p + "g"].T)[..., None]
    return a.reshape(T, -1) @ w[p + "o"].T


def state_space_half(h, w, p, m, eps):
    T, H, P, N, G = len(h), m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = np.split(h @ w[p + "in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, b, c = np.split(xbc, [inner, inner + G * N], axis=1)
    y = state_space_scan(x.reshape(T, H, P), b.reshape(T, G, N), c.reshape(T, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    return gated_group_norm(y.reshape(T, inner), z, m["norm_groups"], w[p + "norm"], eps) @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return m["left_scale"] * attention_half(h, w, p + "left.", m["left"], eps) + \
        m["right_scale"] * state_space_half(h, w, p + "right.", m["right"], eps)


def channel_delta(h, w, p, m, eps):
    T, H, Hk, D, P = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q, k = unit(q.reshape(T, Hk, D)) * D ** -0.5, unit(k.reshape(T, Hk, D))
    beta = sigmoid(h @ w[p + "b"].T)
    step = softplus(h @ w[p + "a1"].T @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(T, H, D)
    decay = np.exp(-np.exp(w[p + "A_log"])[:, None] * step)
    o = rms_norm(delta_scan(q, k, v.reshape(T, H, P), beta, decay), eps, w[p + "norm"])
    gate = sigmoid(h @ w[p + "g1"].T @ w[p + "g2"].T)
    return (o.reshape(T, H * P) * gate) @ w[p + "o"].T


def dense(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg, weights, tokens, dtype=np.float64, read=lambda x: x):
    """(logits [T, vocab], residual after every layer [layers, T, width]).  `read`: what a sublayer sees of the residual, for
    estimates of what rounding alone does."""
    w = {n: np.asarray(a, dtype) for n, a in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x, trace = w["embed"][np.asarray(tokens)], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = {"parallel": parallel, "channel_delta": channel_delta}[layer["type"]]
        x = x + mult * rms_norm(mixer(read(x), w, p + "mix.", layer["mixer"], eps), eps, w[p + "norm1"])
        if layer["mlp"]:
            x = x + mult * rms_norm(dense(read(x), w, p + "mlp."), eps, w[p + "norm2"])
        trace.append(x)
    return read(rms_norm(x, eps, w["final.norm"])) @ w["embed"].T, np.stack(trace)
