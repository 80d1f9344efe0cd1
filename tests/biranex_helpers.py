"""Small random Biranex models for the tests: configuration, weights as the checkpoint names them, and the two ways to run
them (the plain implementation of oracle/biranex.py, and the engine)."""
from __future__ import annotations

import numpy as np
import torch

from oracle import biranex as B
from tests.radivik_helpers import bf16, engine, error, feed, model, status_clear  # noqa: F401  (any registered model)

FP32_LIMIT, BF16_LIMIT = 3e-5, 2e-2


def parallel(heads=4, kv_heads=2, dim=24, vdim=40, window=37, rot_dims=16, base=10000.0, stretch=3.0, scale=0.3, left_scale=0.7,
             ss_heads=6, groups=2, state=20, ss_vdim=12, taps=3, norm_groups=4, right_scale=1.6, ff=40):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window},
            "rot": {"dims": rot_dims, "base": base, "scaling": {"factor": stretch}}}
    right = {"heads": ss_heads, "groups": groups, "state": state, "vdim": ss_vdim, "conv": taps, "norm_groups": norm_groups}
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def delta(heads=6, kv_heads=3, dim=20, vdim=28, taps=4, ff=0, rank_a=9, rank_g=14):
    """rank_a, rank_g: the inner sizes of the two low-rank projections, which only the weights tell."""
    layer = {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps},
             "mlp": {"kind": "dense", "ff": ff} if ff else None}
    RANKS[id(layer)] = (layer, rank_a, rank_g)
    return layer


RANKS: dict[int, tuple] = {}


def config(layers, vocab=97, width=64, mult=0.45, eps=1e-5):
    return {"architecture": "Biranex", "vocab": vocab, "width": width, "residual_mult": mult, "norm": {"eps": eps}, "layers": layers}


def weights(cfg, seed=0, match=0.0):
    """Random weights, exactly representable in bf16.  match > 0: a token 2i + 1 attends every visible token 2i above all
    others.  Its embedding is that of 2i with the halves exchanged, query projections are the group's key projection with the
    columns exchanged in the same way, and `match` scales both norms' weights."""
    g = np.random.default_rng(seed)
    W, w = cfg["width"], {}

    def mat(name, o, i, gain=1.0):
        w[name] = bf16(g.standard_normal((o, i)) * gain * i ** -0.5)

    def vec(name, n, mean=1.0, spread=0.2):
        w[name] = bf16(mean + spread * g.standard_normal(n))

    w["embed"] = bf16(g.standard_normal((cfg["vocab"], W)))
    if match:
        n = cfg["vocab"] // 2
        w["embed"][1 : 2 * n : 2] = np.roll(w["embed"][0 : 2 * n : 2], W // 2, axis=1)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", l["mixer"]
        if l["type"] == "parallel":
            a, s, q, r = m["left"], m["right"], p + "left.", p + "right."
            H, G, D, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            mat(q + "q", H * D, W)
            mat(q + "k", G * D, W)
            mat(q + "v", G * V, W, 2.0)
            vec(q + "q.norm", H * D)
            vec(q + "k.norm", G * D)
            if match:
                k = np.roll(w[q + "k"], W // 2, axis=1).reshape(G, D, W)
                w[q + "q"] = np.repeat(k, H // G, axis=0).reshape(-1, W)
                w[q + "q.norm"], w[q + "k.norm"] = bf16(np.full(H * D, match)), bf16(np.full(G * D, match))
            vec(q + "sink", H, 0.5, 1.0)
            mat(q + "g", H, W, 2.0)
            mat(q + "o", W, H * V)
            inner, bc = s["heads"] * s["vdim"], s["groups"] * s["state"]
            mat(r + "in", 2 * inner + 2 * bc + s["heads"], W, 1.5)
            mat(r + "conv", inner + 2 * bc, s["conv"])
            vec(r + "conv.b", inner + 2 * bc, 0.0, 0.3)
            vec(r + "dt_bias", s["heads"], -0.5, 1.0)
            vec(r + "A_log", s["heads"], -1.5, 1.5)
            vec(r + "D", s["heads"], 0.7, 0.5)
            vec(r + "norm", inner)
            mat(r + "o", W, inner)
        else:
            _, ra, rg = RANKS.get(id(l), (None, 9, 14))
            H, G, D, V, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * V)):
                mat(p + n, rows, W, 1.5)
                mat(p + n + ".conv", rows, T, 1.5)
            mat(p + "b", H, W, 2.0)
            vec(p + "A_log", H, -1.5, 1.2)
            vec(p + "norm", V)
            mat(p + "a1", ra, W)
            mat(p + "a2", H * D, ra)
            vec(p + "dt_bias", H * D, -1.0, 1.0)
            mat(p + "g1", rg, W)
            mat(p + "g2", H * V, rg, 2.0)
            mat(p + "o", W, H * V)
        vec(f"l{i}.norm1", W)
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            mat(f"l{i}.mlp.gate", ff, W, 1.5)
            mat(f"l{i}.mlp.up", ff, W)
            mat(f"l{i}.mlp.down", W, ff)
            vec(f"l{i}.norm2", W)
    vec("final.norm", W)
    return w


def oracle_logits(cfg, w, tokens):
    return B.forward(cfg, w, tokens)[0]


def limits(cfg, w, tokens, want, dtype):
    """Per position: what the logits may differ by.  For bf16, four times what rounding of the sublayers' inputs alone does
    there (a norm behind a sublayer blows rounding up where the sublayer's output happens to be small), or BF16_LIMIT."""
    if dtype == torch.float32:
        return np.full(len(tokens), FP32_LIMIT)
    g = np.random.default_rng(0)
    draws = [error(B.forward(cfg, w, tokens, read=lambda x: bf16(x * (1 + 2.0 ** -9 * g.standard_normal(x.shape))))[0], want) for _ in range(3)]
    return np.maximum(BF16_LIMIT, 4 * np.max(draws, axis=0))


def check(cfg, w, tokens, got, want, dtype):
    """`got`: one or several runs of the tokens' logits."""
    top = limits(cfg, w, tokens, want, dtype)
    for g in got if isinstance(got, list) else [got]:
        err = error(g, want)
        assert (err < top).all(), [(int(i), err[i], top[i]) for i in np.nonzero(err >= top)[0][:5]]


CONFIGS = {
    "small": config([parallel(), delta(), parallel(heads=3, kv_heads=3, dim=40, vdim=16, rot_dims=8, window=64, ss_heads=4, groups=4, state=12,
                                                   ss_vdim=20, taps=4, norm_groups=1, ff=0), delta(ff=24)]),
    # sizes the tensor-core kernels take without padding; a window that is no multiple of a page
    "wide": config([parallel(heads=8, kv_heads=2, dim=128, vdim=64, window=70, rot_dims=128, ss_heads=4, groups=1, state=64, ss_vdim=64,
                             norm_groups=1, taps=4, ff=96, scale=0.09), delta(heads=4, kv_heads=4, dim=64, vdim=64, taps=2, rank_a=16,
                                                                              rank_g=24)], vocab=130, width=128, mult=0.8),
    # nothing is a multiple of anything
    "odd": config([parallel(heads=3, kv_heads=1, dim=10, vdim=7, window=5, rot_dims=4, stretch=1.0, ss_heads=3, groups=1, state=5, ss_vdim=7,
                            norm_groups=7, taps=5, ff=9), delta(heads=2, kv_heads=1, dim=9, vdim=11, taps=3, ff=7, rank_a=5, rank_g=3)],
                  vocab=51, width=30, mult=1.0, eps=1e-6),
    # everything that can be 1 is 1; the window shows a token itself alone
    "ones": config([parallel(heads=1, kv_heads=1, dim=8, vdim=8, window=1, rot_dims=2, ss_heads=1, groups=1, state=4, ss_vdim=8, norm_groups=1,
                             taps=1, ff=8), delta(heads=1, kv_heads=1, dim=4, vdim=4, taps=1, rank_a=1, rank_g=1)], vocab=40, width=32),
    # heads too large for the tensor-core attention and for one block's registers of state
    "large_heads": config([parallel(heads=2, kv_heads=1, dim=160, vdim=136, window=33, rot_dims=64, ss_heads=2, groups=2, state=144, ss_vdim=136,
                                    norm_groups=2, ff=0), delta(heads=2, kv_heads=2, dim=136, vdim=264, taps=6, rank_a=8, rank_g=8)], width=96),
}


def prompt(n, vocab, seed=0):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def far_prompt(n, vocab, seed=0, window=37):
    """Random tokens, and rare ones whose counterparts (2i, then 2i + 1) come back at the end, around page borders, and just
    inside and just outside a window."""
    p = np.random.default_rng(seed).integers(10, vocab, n)
    for at, tok in ((0, 0), (2, 0), (14, 2), (17, 4), (60, 4), (65, 6), (n // 2, 8)):
        for d, t in ((0, tok), (window - 1, tok + 1), (window, tok + 1)):
            if at + d < n:
                p[at + d] = t
    p[-3:] = [5, 7, 9][-min(n, 3):]
    return p.tolist()
