"""Biranex: a decoder with a 32-bit residual stream and norms on the sublayers' outputs only, whose layers are of two kinds:

    parallel       windowed grouped-query attention and a Mamba-2 layer side by side on the same input (Dao and Gu,
                   "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State Space
                   Duality"): norm of the whole query and key projections, interleaved rotation with linear scaling, a sink
                   in the softmax, a gate per head; the two results are scaled and added
    channel_delta  a gated delta rule with one decay per head and key channel

One layer, x the residual row:
    x <- x + m norm1(mixer(x))
    x <- x + m norm2(W_down(silu(W_gate x) * W_up x))     (not in every layer)
The residual, the norms, angles, scores and softmax, the recurrent states and all that enters them behind the projections and
convolutions are 32-bit; products run in the model's precision.  The head is the embedding table.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import kernels as K
from .. import ops
from ..checkpoint import RandomWeights
from . import StepOutput, register

UNIT_EPS = 1e-6  # in the unit norm of the delta rule's queries and keys


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rotary: ops.Rotary | None
    window: int  # 0: none


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    groups: int
    state: int
    vdim: int
    taps: int
    norm_groups: int


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    right: StateSpaceConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class LayerConfig:
    mixer: ParallelConfig | DeltaConfig
    ff: int  # 0: no feed-forward


@dataclass(frozen=True)
class BiranexConfig:
    vocab: int
    width: int
    mult: float
    eps: float
    layers: tuple[LayerConfig, ...]

    @classmethod
    def from_dict(cls, c: dict) -> "BiranexConfig":
        layers = []
        for i, layer in enumerate(c["layers"]):
            where, m = f"layer {i}", layer["mixer"]
            if layer["type"] == "parallel":
                mixer = ParallelConfig(read_attention(m["left"], where), read_state_space(m["right"], where), float(m["left_scale"]),
                                       float(m["right_scale"]))
            elif layer["type"] == "channel_delta":
                grouped(m["heads"], m["kv_heads"], where)
                mixer = DeltaConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
            else:
                raise ValueError(f"{where}: unknown mixer {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"{where}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerConfig(mixer, mlp["ff"] if mlp else 0))
        return cls(c["vocab"], c["width"], float(c["residual_mult"]), float(c["norm"]["eps"]), tuple(layers))


def grouped(heads: int, groups: int, where: str) -> None:
    if groups < 1 or heads < 1 or heads % groups:
        raise ValueError(f"{where}: {heads} heads over {groups}")


def read_attention(m: dict, where: str) -> AttentionConfig:
    grouped(m["heads"], m["kv_heads"], where)
    rot, rotary = m.get("rot"), None
    if rot and rot["dims"] > 0:
        if rot["dims"] % 2 or rot["dims"] > m["dim"]:
            raise ValueError(f"{where}: rotation of {rot['dims']} of {m['dim']} channels")
        rotary = ops.Rotary(rot["dims"], float(rot["base"]), stretch=float((rot.get("scaling") or {}).get("factor", 1.0)))
    window = (m.get("mask") or {}).get("size") or 0
    if window < 0:
        raise ValueError(f"{where}: window of {window}")
    return AttentionConfig(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), rotary, window)


def read_state_space(m: dict, where: str) -> StateSpaceConfig:
    grouped(m["heads"], m["groups"], where)
    grouped(m["heads"] * m["vdim"], m["norm_groups"], where)
    return StateSpaceConfig(m["heads"], m["groups"], m["state"], m["vdim"], m["conv"], m["norm_groups"])


class Loader:
    """Takes a layer's tensors from the weights: matrices as stored, everything that works in 32-bit as fp32 on the device."""

    def __init__(self, weights, device, dtype):
        self.weights, self.device, self.dtype = weights, device, dtype

    def mat(self, name: str, *shape: int) -> torch.Tensor:
        return self.weights.take(name, *shape)

    def f32(self, name: str, *shape: int) -> torch.Tensor:
        return self.weights.take(name, *shape).to(self.device, torch.float32).contiguous()

    def taps(self, name: str, channels: int, taps: int) -> torch.Tensor:
        """[taps, channels]: a token's products with one tap lie side by side."""
        return self.f32(name, channels, taps).t().contiguous()


class ParallelMixer:
    """Left and right read one product of the input; their outputs lie side by side in front of one product, whose columns
    are both output matrices.  The two scales are applied in 32-bit before: left in the attention's last step, right in
    the norm's."""

    def __init__(self, ld: Loader, p: str, c: ParallelConfig, width: int, eps: float):
        a, s = c.left, c.right
        inner, bc = s.heads * s.vdim, s.groups * s.state
        q, k = p + "left.", p + "right."
        w_in = ld.mat(k + "in", 2 * inner + 2 * bc + s.heads, width)
        self.cfg, self.eps = c, eps
        self.proj = ops.Packed({
            "qkv": torch.cat([ld.mat(q + "q", a.heads * a.dim, width), ld.mat(q + "k", a.kv_heads * a.dim, width),
                              ld.mat(q + "v", a.kv_heads * a.vdim, width)]),
            "g": ld.mat(q + "g", a.heads, width), "z": w_in[:inner], "xbc": w_in[inner : 2 * inner + 2 * bc],
            "dt": w_in[2 * inner + 2 * bc :]}, ld.dtype, ld.device)
        self.q_norm, self.k_norm = ld.f32(q + "q.norm", a.heads * a.dim), ld.f32(q + "k.norm", a.kv_heads * a.dim)
        self.sink = ld.f32(q + "sink", a.heads)
        self.rec = ops.Recurrence(
            s.heads, s.groups, s.state, s.vdim, ld.taps(k + "conv", inner + 2 * bc, s.taps), ld.f32(k + "conv.b", inner + 2 * bc),
            -ld.f32(k + "A_log", s.heads).exp(), ld.f32(k + "dt_bias", s.heads), ld.f32(k + "D", s.heads),
            off_q=inner + bc, off_k=inner, off_v=0)
        self.norm = ops.GatedNorm(ld.f32(k + "norm", inner), s.norm_groups, eps, gate_first=True, out_scale=c.right_scale)
        left, right = ld.mat(q + "o", width, a.heads * a.vdim), ld.mat(k + "o", width, inner)
        # columns behind each half up to a multiple of 8 are zero on both sides
        self.left_cols, self.right_at = left.shape[1], (left.shape[1] + 7) // 8 * 8
        cols = self.right_at + (inner + 7) // 8 * 8
        self.padded = cols != left.shape[1] + inner
        self.out = torch.zeros(width, cols, dtype=ld.dtype, device=ld.device)
        self.out[:, : self.left_cols] = left.to(ld.device, ld.dtype)
        self.out[:, self.right_at : self.right_at + inner] = right.to(ld.device, ld.dtype)
        self.inner = inner

    def make_cache(self, num_pages, page_size, slots, dtype, device):
        a = self.cfg.left
        return (ops.make_paged_kv(num_pages, a.kv_heads, page_size, a.dim, a.vdim, dtype, device),
                ops.make_recurrent_state(self.rec, slots, dtype, device))

    def __call__(self, xb: torch.Tensor, rows: ops.Rows, cache, tables) -> torch.Tensor:
        a, (kv, state), N = self.cfg.left, cache, xb.shape[0]
        y = self.proj(xb)
        part = lambda name: self.proj.part(y, name)  # noqa: E731
        both = (torch.zeros if self.padded else torch.empty)(N, self.out.shape[1], dtype=xb.dtype, device=xb.device)
        q = ops.norm_rope_write(part("qkv"), rows, kv, self.q_norm, self.k_norm, self.eps, tables.get(a.rotary), a.heads)
        left = both[:, : self.left_cols].unflatten(1, (a.heads, a.vdim))
        ops.paged_attention(q, kv, rows, a.scale, ops.AttnOptions(a.window, self.sink, part("g"), self.cfg.left_scale), left)
        ops.recurrent_mixer(self.rec, state, part("xbc"), part("dt"), None, part("z"), self.norm, rows,
                            both[:, self.right_at : self.right_at + self.inner])
        return K.linear(both, self.out)


class DeltaMixer:
    def __init__(self, ld: Loader, p: str, c: DeltaConfig, width: int, eps: float):
        qk, v = c.kv_heads * c.dim, c.heads * c.vdim
        rank_a, rank_g = (ld.weights.shape(p + n, (size, width))[0] for n, size in (("a1", c.dim), ("g1", c.vdim)))
        self.cfg = c
        self.proj = ops.Packed({
            "x": torch.cat([ld.mat(p + "q", qk, width), ld.mat(p + "k", qk, width), ld.mat(p + "v", v, width)]),
            "b": ld.mat(p + "b", c.heads, width), "a1": ld.mat(p + "a1", rank_a, width), "g1": ld.mat(p + "g1", rank_g, width)},
            ld.dtype, ld.device)
        self.a2 = ld.mat(p + "a2", c.heads * c.dim, rank_a).to(ld.device, ld.dtype)
        self.g2 = ld.mat(p + "g2", v, rank_g).to(ld.device, ld.dtype)
        conv = torch.cat([ld.taps(p + "q.conv", qk, c.taps), ld.taps(p + "k.conv", qk, c.taps), ld.taps(p + "v.conv", v, c.taps)], dim=1)
        self.rec = ops.Recurrence(
            c.heads, c.kv_heads, c.dim, c.vdim, conv, None, -ld.f32(p + "A_log", c.heads).exp(), ld.f32(p + "dt_bias", c.heads * c.dim),
            None, off_q=0, off_k=qk, off_v=2 * qk, channel_decay=True, correct=True, unit_eps=UNIT_EPS, q_scale=c.dim ** -0.5)
        self.norm = ops.GatedNorm(ld.f32(p + "norm", c.vdim), c.heads, eps, gate_first=False)
        self.out = ld.mat(p + "o", width, v).to(ld.device, ld.dtype)

    def make_cache(self, num_pages, page_size, slots, dtype, device):
        return ops.make_recurrent_state(self.rec, slots, dtype, device)

    def __call__(self, xb: torch.Tensor, rows: ops.Rows, cache, tables) -> torch.Tensor:
        y = self.proj(xb)
        part = lambda name: self.proj.part(y, name)  # noqa: E731
        step, gate = K.linear(part("a1"), self.a2), K.linear(part("g1"), self.g2)
        o = torch.empty(xb.shape[0], self.out.shape[1], dtype=xb.dtype, device=xb.device)
        ops.recurrent_mixer(self.rec, cache, part("x"), step, part("b"), gate, self.norm, rows, o)
        return K.linear(o, self.out)


@dataclass
class Layer:
    mixer: ParallelMixer | DeltaMixer
    norm1: torch.Tensor
    norm2: torch.Tensor | None
    gate_up: torch.Tensor | None  # gate rows | up rows
    down: torch.Tensor | None
    ff: int


@register("Biranex")
class Biranex:
    page_size = 64  # one tensor-map box of a key block; the engine's default for this model
    stateful = True  # keeps a state per request beside the pages: the engine hands out slots

    def __init__(self, cfg: BiranexConfig, weights, device, dtype: torch.dtype = torch.bfloat16):
        """`weights.take(name, *shape)` yields host or device tensors (checkpoint.Weights or RandomWeights)."""
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"unsupported precision {dtype}")
        if dtype == torch.float32:  # true 32-bit products
            torch.backends.cuda.matmul.allow_tf32 = False
        self.cfg, self.device, self.dtype = cfg, device, dtype
        self.vocab, self.width, self.num_layers = cfg.vocab, cfg.width, len(cfg.layers)
        self.tau = 0.0
        self.seed = torch.zeros(1, dtype=torch.int64, device=device)
        W, ld = cfg.width, Loader(weights, device, dtype)
        self.embed = ld.mat("embed", cfg.vocab, W).to(device, dtype)  # also the head
        self.layers = []
        for i, lc in enumerate(cfg.layers):
            p = f"l{i}."
            kind = ParallelMixer if isinstance(lc.mixer, ParallelConfig) else DeltaMixer
            layer = Layer(kind(ld, p + "mix.", lc.mixer, W, cfg.eps), ld.f32(p + "norm1", W), None, None, None, lc.ff)
            if lc.ff:
                layer.norm2 = ld.f32(p + "norm2", W)
                layer.gate_up = torch.cat([ld.mat(p + "mlp.gate", lc.ff, W), ld.mat(p + "mlp.up", lc.ff, W)]).to(device, dtype)
                layer.down = ld.mat(p + "mlp.down", W, lc.ff).to(device, dtype)
            self.layers.append(layer)
        self.norm = ld.f32("final.norm", W)
        self.tables: dict[ops.Rotary, torch.Tensor] = {}

    @classmethod
    def from_config(cls, config: dict, weights, device, dtype: torch.dtype = torch.bfloat16) -> "Biranex":
        cfg = BiranexConfig.from_dict(config)
        return cls(cfg, RandomWeights(device) if weights is None else weights, device, dtype)

    # ------------------------------------------------------------------ what the engine drives
    def make_caches(self, num_pages: int, page_size: int, max_len: int, slots: int) -> list:
        """Per layer: pages and a state per slot (parallel), or the state alone (delta); and the tables of positions."""
        for c in self.cfg.layers:
            r = c.mixer.left.rotary if isinstance(c.mixer, ParallelConfig) else None
            if r is not None and (r not in self.tables or self.tables[r].shape[0] < max_len):
                self.tables[r] = r.table(max_len, self.device)
        return [L.mixer.make_cache(num_pages, page_size, slots, self.dtype, self.device) for L in self.layers]

    def make_prefix(self, max_len: int) -> None:
        return None  # attention reads the cache by page

    @torch.inference_mode()
    def step(self, caches, inp, ids, cached_lens, block_table, num_decoding, prefix=None, slots=None, trace: list | None = None) -> StepOutput:
        """One step; `inp is None` = pure decode.  `trace`: receives a copy of the residual after every layer."""
        rows = ops.Rows(ids.shape[0], cached_lens, num_decoding, block_table, slots=slots)
        if inp is not None:
            rows.seq_ids, rows.positions, rows.cu_seqlens = inp.seq_ids, inp.positions, inp.cu_seqlens
            rows.tile_start, rows.block_m = inp.tile_start, inp.block_m
        c, dt = self.cfg, self.dtype
        x, xb = ops.embed(self.embed, ids)
        for L, cache in zip(self.layers, caches):
            xb = ops.norm_add(x, L.mixer(xb, rows, cache, self.tables), L.norm1, c.mult, c.eps, dt)
            if L.ff:
                h = ops.silu_mul(K.linear(xb, L.gate_up), L.ff)
                xb = ops.norm_add(x, K.linear(h, L.down), L.norm2, c.mult, c.eps, dt)
            if trace is not None:
                trace.append(x.clone())
        _, hidden = ops.scaled_add_norm(x, None, self.norm, 1.0, c.eps, dt, keep=False)
        last = hidden if inp is None else hidden[(inp.cu_seqlens[1:] - 1).clamp(min=0).long()]
        return StepOutput(K.sample(self.logits(last), self.tau, self.seed).view(-1), hidden)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return K.linear(hidden, self.embed, out_dtype=torch.float32)
