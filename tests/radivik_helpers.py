"""Small random Radivik models for the tests: configuration, weights as the checkpoint names them, and the two ways to run
them (the plain implementation of oracle/radivik.py, and the engine)."""
from __future__ import annotations

import numpy as np
import torch

from oracle import radivik as R


def layer(heads=4, kv_heads=2, dim=48, vdim=40, rot_dims=16, base=10000.0, scaling=None, scale=None, kv_from=None, experts=4, top=2,
          ff=40, limit=2.0, mlp=True):
    rot = {"dims": rot_dims, "base": base}
    if scaling:
        rot["scaling"] = scaling
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": dim ** -0.5 if scale is None else scale}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    out = {"type": "attention", "mixer": mixer, "mlp": None}
    if mlp:
        out["mlp"] = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    return out


YARN = {"factor": 8.0, "original": 64, "fast": 8.0, "slow": 1.0}


def config(layers, vocab=97, width=64, alpha=1.7, eps=1e-5):
    return {"architecture": "Radivik", "vocab": vocab, "width": width, "postln_alpha": alpha, "norm": {"eps": eps}, "layers": layers}


def small(scale=None, **kw):
    """Three layers that differ: scaled rotation and two experts a token; a layer on the first one's cache; plain rotation,
    no feed-forward."""
    return config([layer(scaling=YARN, scale=scale), layer(kv_from=0, heads=6, experts=5, top=1, ff=24, limit=0.7, scaling=YARN, scale=scale),
                   layer(rot_dims=8, heads=3, kv_heads=3, dim=24, vdim=56, mlp=False, scale=scale)], **kw)


def bf16(x):
    return torch.tensor(np.asarray(x, np.float32)).to(torch.bfloat16).float().numpy()


def weights(cfg, seed=0, match=False):
    """Random weights, exactly representable in bf16.  match: query and key projections of a group are equal, so that a
    token attends its own earlier occurrences, wherever they are."""
    g = np.random.default_rng(seed)
    W, w = cfg["width"], {}

    def mat(name, o, i, gain=1.0):
        w[name] = bf16(g.standard_normal((o, i)) * gain * i ** -0.5)

    def norm(name):
        w[name] = bf16(1.0 + 0.2 * g.standard_normal(W))

    w["embed"] = bf16(g.standard_normal((cfg["vocab"], W)))
    own = {}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        src = m.get("kv_from")
        mat(p + "mix.q", m["heads"] * m["dim"], W)
        if src is None:
            mat(p + "mix.k", m["kv_heads"] * m["dim"], W)
            mat(p + "mix.v", m["kv_heads"] * m["vdim"], W)
            own[i] = w[p + "mix.k"]
        if match:
            k = own[i if src is None else src].reshape(m["kv_heads"], m["dim"], W)
            w[p + "mix.q"] = np.repeat(k, m["heads"] // m["kv_heads"], axis=0).reshape(-1, W)
        mat(p + "mix.o", W, m["heads"] * m["vdim"])
        norm(p + "norm1")
        if l["mlp"]:
            r, e = l["mlp"]["router"], l["mlp"]["expert"]
            mat(p + "mlp.router", r["experts"], W)
            for n in range(r["experts"]):
                q = f"{p}mlp.e{n}."
                mat(q + "gate", e["ff"], W, 3.0)
                mat(q + "up", e["ff"], W, 3.0)
                mat(q + "down", W, e["ff"])
            norm(p + "norm2")
    norm("final.norm")
    mat("head", cfg["vocab"], W)
    return w


def model(cfg, w, dtype=torch.float32):
    from inference_engine_b200.checkpoint import Weights
    from inference_engine_b200.models import model_class

    src = Weights({k: torch.tensor(v).to(torch.bfloat16) for k, v in w.items()})
    m = model_class(cfg).from_config(cfg, src, torch.device("cuda", 0), dtype)
    assert src.unused() == []
    return m


def engine(m, max_batch=4, max_len=512, page_size=16, graphs=False, **kw):
    from inference_engine_b200.engine import Engine

    args = dict(max_tokens_per_step=max_len + max_batch, min_first_chunk=16, max_graph_tokens=64)
    args.update(kw)
    return Engine(m, max_batch, max_len, -1, page_size=page_size, use_graphs=graphs, **args)


def feed(eng, tokens, cuts):
    """Logits of every token, fed as one request in portions that end at `cuts` and at the end."""
    r = eng.open_replay()
    out, at = [], 0
    for end in [c for c in cuts if c < len(tokens)] + [len(tokens)]:
        part = tokens[at:end]
        out.append(eng.replay([(r, part, list(range(len(part))))]).numpy())
        at = end
    eng.close_replay(r)
    return np.concatenate(out)


def error(got, want):
    """Per position: the logits' difference, mean taken off, over the spread of the logits."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=1, keepdims=True)
    spread = np.sqrt(((want - want.mean(axis=1, keepdims=True)) ** 2).mean())
    return np.sqrt((d ** 2).mean(axis=1)) / spread


TOLERANCE = {torch.float32: 2e-5, torch.bfloat16: 4e-2}


def oracle_logits(cfg, w, tokens):
    return R.forward(cfg, w, tokens)[0]


def settle(cfg, w, tokens, least=0.01):
    """The prompt with tokens exchanged until no router is within `least` of choosing otherwise, so that rounding cannot turn
    a choice (two experts' outputs have nothing in common, and one turned choice would hide everything else)."""
    tokens, g = list(tokens), np.random.default_rng(len(tokens))
    for _ in range(600):
        margins = []
        R.forward(cfg, w, tokens, margins=margins)
        close = np.nonzero(np.min(margins, axis=0) < least)[0] if margins else []
        if len(close) == 0:
            return tokens
        for at in close[:3]:
            tokens[at] = int(g.integers(0, cfg["vocab"]))
    raise AssertionError("no settled prompt found")


def status_clear():
    from inference_engine_b200 import kernels as K

    assert K.check_status() == 0
