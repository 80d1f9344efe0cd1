"""Radivik: a decoder with a 32-bit residual stream normed after every sum, grouped-query attention with unit-norm
rotated heads (key and value sizes free of one another, layers may attend an earlier layer's cache), and a mixture of
experts whose scores scale the experts' inputs.

One layer, x the residual row:
    x <- norm1(alpha x + O attend(q, K, V))      q, k = unit(rotate(W x)), v = W x
    x <- norm2(alpha x + sum_e expert_e(s_e x))  s = sigmoid(router x), the `top` largest
The residual, the norms, the rotation, scores and softmax and the router are 32-bit; products run in the model's
precision.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import kernels as K
from .. import ops
from ..checkpoint import RandomWeights
from . import StepOutput, register

GATE_SLOPE = 1.702  # y = g * sigmoid(slope * g) * (u + 1)


@dataclass(frozen=True)
class MixerConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rotary: ops.Rotary | None
    kv_from: int | None


@dataclass(frozen=True)
class MlpConfig:
    experts: int
    top: int
    ff: int
    limit: float


@dataclass(frozen=True)
class LayerConfig:
    mixer: MixerConfig
    mlp: MlpConfig | None


@dataclass(frozen=True)
class RadivikConfig:
    vocab: int
    width: int
    alpha: float
    eps: float
    layers: tuple[LayerConfig, ...]

    @classmethod
    def from_dict(cls, c: dict) -> "RadivikConfig":
        layers = []
        for i, layer in enumerate(c["layers"]):
            if layer["type"] != "attention":
                raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
            mixer = read_mixer(layer["mixer"], f"layer {i}")
            src = mixer.kv_from
            if src is not None:
                if not 0 <= src < i or layers[src].mixer.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from {src} is not an earlier layer with keys of its own")
                own = layers[src].mixer
                if (own.kv_heads, own.dim, own.vdim) != (mixer.kv_heads, mixer.dim, mixer.vdim):
                    raise ValueError(f"layer {i}: its heads differ from those of layer {src}, whose cache it uses")
            layers.append(LayerConfig(mixer, read_mlp(layer.get("mlp"), f"layer {i}")))
        return cls(c["vocab"], c["width"], float(c["postln_alpha"]), float(c["norm"]["eps"]), tuple(layers))


def read_mixer(m: dict, where: str) -> MixerConfig:
    heads, kv = m["heads"], m["kv_heads"]
    if kv < 1 or heads % kv:
        raise ValueError(f"{where}: {heads} query heads over {kv} key/value heads")
    rot = m.get("rot")
    rotary = None
    if rot and rot["dims"] > 0:
        if rot["dims"] % 2 or rot["dims"] > m["dim"]:
            raise ValueError(f"{where}: rotation of {rot['dims']} of {m['dim']} channels")
        sc = rot.get("scaling")
        scaling = None if not sc else (float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"]))
        rotary = ops.Rotary(rot["dims"], float(rot["base"]), scaling)
    return MixerConfig(heads, kv, m["dim"], m["vdim"], float(m["scale"]), rotary, m.get("kv_from"))


def read_mlp(m: dict | None, where: str) -> MlpConfig | None:
    if not m:
        return None
    if m.get("kind", "moe") != "moe":
        raise ValueError(f"{where}: unknown feed-forward {m['kind']!r}")
    r, e = m["router"], m["expert"]
    if not 1 <= r["top"] <= r["experts"]:
        raise ValueError(f"{where}: top {r['top']} of {r['experts']} experts")
    return MlpConfig(r["experts"], r["top"], e["ff"], float(e["limit"]))


@dataclass
class Layer:
    cfg: LayerConfig
    cache: int  # index of the layer whose cache it uses
    qkv: torch.Tensor  # q | k | v rows (q only with kv_from)
    o: torch.Tensor
    norm1: torch.Tensor
    norm2: torch.Tensor | None
    experts: ops.Experts | None


@register("Radivik")
class Radivik:
    page_size = 64  # one tensor-map box of a key block; the engine's default for this model

    def __init__(self, cfg: RadivikConfig, weights, device, dtype: torch.dtype = torch.bfloat16):
        """`weights.take(name, *shape)` yields host or device tensors (checkpoint.Weights or RandomWeights)."""
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"unsupported precision {dtype}")
        if dtype == torch.float32:  # true 32-bit products
            torch.backends.cuda.matmul.allow_tf32 = False
        self.cfg, self.device, self.dtype = cfg, device, dtype
        self.vocab, self.width, self.num_layers = cfg.vocab, cfg.width, len(cfg.layers)
        self.tau = 0.0
        self.seed = torch.zeros(1, dtype=torch.int64, device=device)
        take, W = weights.take, cfg.width

        def norm(name):
            return take(name, W).to(device, torch.float32)

        self.embed = take("embed", cfg.vocab, W).to(device, dtype)
        self.layers = []
        for i, lc in enumerate(cfg.layers):
            p, m = f"l{i}.", lc.mixer
            parts = [take(p + "mix.q", m.heads * m.dim, W)]
            if m.kv_from is None:
                parts += [take(p + "mix.k", m.kv_heads * m.dim, W), take(p + "mix.v", m.kv_heads * m.vdim, W)]
            experts = None
            if lc.mlp:
                f = lc.mlp
                e = [p + f"mlp.e{n}." for n in range(f.experts)]
                experts = ops.make_experts(
                    take(p + "mlp.router", f.experts, W), [take(n + "gate", f.ff, W) for n in e], [take(n + "up", f.ff, W) for n in e],
                    [take(n + "down", W, f.ff) for n in e], f.top, f.limit, GATE_SLOPE, dtype, device)
            self.layers.append(Layer(
                lc, i if m.kv_from is None else m.kv_from, torch.cat([t.to(device, dtype) for t in parts]),
                take(p + "mix.o", W, m.heads * m.vdim).to(device, dtype), norm(p + "norm1"), norm(p + "norm2") if lc.mlp else None, experts))
        self.norm = norm("final.norm")
        self.head = take("head", cfg.vocab, W).to(device, dtype)
        self.tables: dict[ops.Rotary, torch.Tensor] = {}

    @classmethod
    def from_config(cls, config: dict, weights, device, dtype: torch.dtype = torch.bfloat16) -> "Radivik":
        cfg = RadivikConfig.from_dict(config)
        return cls(cfg, RandomWeights(device) if weights is None else weights, device, dtype)

    # ------------------------------------------------------------------ what the engine drives
    def make_caches(self, num_pages: int, page_size: int, max_len: int) -> list[ops.PagedKV | None]:
        """One paged cache per layer that has keys of its own (None for the others), and the tables of positions."""
        for L in self.layers:
            r = L.cfg.mixer.rotary
            if r is not None and (r not in self.tables or self.tables[r].shape[0] < max_len):
                self.tables[r] = r.table(max_len, self.device)
        return [None if L.cfg.mixer.kv_from is not None else
                ops.make_paged_kv(num_pages, L.cfg.mixer.kv_heads, page_size, L.cfg.mixer.dim, L.cfg.mixer.vdim, self.dtype, self.device)
                for L in self.layers]

    def make_prefix(self, max_len: int) -> None:
        return None  # attention reads the cache by page

    @torch.inference_mode()
    def step(self, caches, inp, ids, cached_lens, block_table, num_decoding, prefix=None, trace: list | None = None) -> StepOutput:
        """One step; `inp is None` = pure decode.  `trace`: receives a copy of the residual after every layer."""
        if inp is None:
            rows = ops.Rows(ids.shape[0], cached_lens, num_decoding, block_table)
        else:
            rows = ops.Rows(ids.shape[0], cached_lens, num_decoding, block_table, inp.seq_ids, inp.positions, inp.cu_seqlens,
                            inp.tile_start, inp.block_m)
        c, dt = self.cfg, self.dtype
        x, xb = ops.embed(self.embed, ids)
        for L in self.layers:
            m, cache = L.cfg.mixer, caches[L.cache]
            q = ops.rope_write(K.linear(xb, L.qkv), rows, cache, self.tables[m.rotary] if m.rotary else None, m.heads,
                               m.kv_from is None, True, c.eps)
            a = ops.paged_attention(q, cache, rows, m.scale)
            y = K.linear(a.view(rows.num_rows, m.heads * m.vdim), L.o)
            x, xb = ops.scaled_add_norm(x, y, L.norm1, c.alpha, c.eps, dt, zero=L.experts.counts if L.experts else None)
            if L.experts:
                y, places = ops.mixture(x, xb, L.experts)
                x, xb = ops.scaled_add_norm(x, y, L.norm2, c.alpha, c.eps, dt, index=places)
            if trace is not None:
                trace.append(x.clone())
        _, hidden = ops.scaled_add_norm(x, None, self.norm, 1.0, c.eps, dt, keep=False)
        last = hidden if inp is None else hidden[(inp.cu_seqlens[1:] - 1).clamp(min=0).long()]
        return StepOutput(K.sample(self.logits(last), self.tau, self.seed).view(-1), hidden)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return K.linear(hidden, self.head, out_dtype=torch.float32)
