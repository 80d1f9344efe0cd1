"""Decoder ops in the model's own precision (bf16 or fp32), over libb200dec.so (include/b200dec.h).

They stand beside `kernels` (the int8-cache attention path with the reference's signatures) and cover what a decoder of
another design needs: a paged KV cache of unquantised rows whose key and value sizes are free of one another, partial
rotary positions with frequency scaling, unit-norm heads, a 32-bit residual stream normed after the sum, and a mixture of
experts.  Every constant of a design is an argument.  As in `kernels` there is no CPU path: CPU tensors raise.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from . import _lib
from . import kernels as K

MAX_TENSOR_CORE_DIM = 128  # head sizes up to this run on the tensor-core attention kernels (bf16)


def _lib_dec():
    lib = _lib.load_decoder()
    if K._early_start and not lib.b200kv_get_chained_launch():
        lib.b200kv_set_chained_launch(1)
    return lib


def _ptr(t: torch.Tensor | None):
    return None if t is None else t.data_ptr()


def _elem(dtype: torch.dtype) -> int:
    if dtype not in (torch.bfloat16, torch.float32):
        raise ValueError(f"decoder ops run in bfloat16 or float32, not {dtype}")
    return 2 if dtype == torch.bfloat16 else 4


def _round8(n: int) -> int:
    return (n + 7) // 8 * 8


# ----------------------------------------------------------------------------- the paged cache of unquantised rows
@dataclass
class PagedKV:
    """One layer's keys and values, rows padded to 8 channels (the padding stays zero)."""

    k: torch.Tensor  # [num_pages, kv_heads, page_size, round8(k_dim)]
    v: torch.Tensor  # [num_pages, kv_heads, page_size, round8(v_dim)]
    k_dim: int
    v_dim: int

    @property
    def kv_heads(self) -> int:
        return self.k.shape[1]

    @property
    def page_size(self) -> int:
        return self.k.shape[2]

    def struct(self) -> _lib.DecCache:
        k, v = self.k, self.v
        return _lib.DecCache(k.data_ptr(), v.data_ptr(), k.shape[0], k.shape[1], k.shape[2], self.k_dim, self.v_dim, k.shape[3],
                             v.shape[3], k.element_size())


def make_paged_kv(num_pages: int, kv_heads: int, page_size: int, k_dim: int, v_dim: int, dtype, device) -> PagedKV:
    def z(d):
        return torch.zeros(num_pages, kv_heads, page_size, _round8(d), dtype=dtype, device=device)

    return PagedKV(z(k_dim), z(v_dim), k_dim, v_dim)


@dataclass
class Rows:
    """Which (entry, position) each packed row of a step is.  seq_ids / positions None: pure decode, row = entry at
    position cached_lens[row], rows from num_decoding on idle."""

    num_rows: int
    cached_lens: torch.Tensor
    num_decoding: torch.Tensor
    block_table: torch.Tensor  # int32 [entries, max_pages]
    seq_ids: torch.Tensor | None = None
    positions: torch.Tensor | None = None
    cu_seqlens: torch.Tensor | None = None
    tile_start: torch.Tensor | None = None
    block_m: int = 128
    slots: torch.Tensor | None = None  # int32 [entries]: state slots of recurrent layers, -1 = passed over

    def struct(self) -> _lib.DecRows:
        return _lib.DecRows(_ptr(self.seq_ids), _ptr(self.positions), K._i32(self.cached_lens), K._i32(self.num_decoding),
                            self.num_rows)

    def entries(self) -> _lib.Entries:
        return _lib.Entries(_ptr(self.cu_seqlens), K._i32(self.cached_lens), K._i32(self.num_decoding), K._i32(self.slots),
                            _ptr(self.seq_ids), _ptr(self.positions), self.cached_lens.shape[0], self.num_rows)


# ----------------------------------------------------------------------------- rotary positions
@dataclass(frozen=True)
class Rotary:
    """Rotation of the first `dims` channels of a head, channel i paired with i + dims / 2 (rope_write) or 2i with 2i + 1
    (norm_rope_write).  With `scaling` (factor,
    original, fast, slow) the frequencies are stretched as YaRN does (Peng et al., "YaRN: Efficient Context Window
    Extension of Large Language Models"): components that turn more than `fast` times within the original context
    keep their frequency, those that turn less than `slow` times are divided by `factor`, a linear ramp joins the two,
    and cos and sin are multiplied by 0.1 ln(factor) + 1."""

    dims: int
    base: float
    scaling: tuple[float, float, float, float] | None = None  # factor, original, fast, slow
    stretch: float = 1.0  # linear scaling: every frequency is divided by it

    def frequencies(self) -> tuple[list[float], float]:
        half = self.dims // 2
        freq = [self.base ** (-2.0 * i / self.dims) / self.stretch for i in range(half)]
        if self.scaling is None:
            return freq, 1.0
        factor, original, fast, slow = self.scaling

        def component(turns: float) -> float:
            return self.dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))

        lo = max(math.floor(component(fast)), 0)
        hi = min(math.ceil(component(slow)), self.dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(half)]
        return [f / factor * r + f * (1.0 - r) for f, r in zip(freq, ramp)], 0.1 * math.log(factor) + 1.0

    def table(self, length: int, device) -> torch.Tensor:
        """fp32 [length, dims / 2, 2]: cos and sin of every position, multiplier included (angles in 64-bit)."""
        freq, mult = self.frequencies()
        pos = torch.arange(length, dtype=torch.float64, device=device)
        a = pos[:, None] * torch.tensor(freq, dtype=torch.float64, device=device)
        return (torch.stack((a.cos(), a.sin()), dim=-1) * mult).to(torch.float32).contiguous()


# ----------------------------------------------------------------------------- row ops
@K._ranged
def embed(table: torch.Tensor, ids: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
    """(residual rows fp32, the same rows in the model's precision; one tensor when that is fp32)."""
    K._require_cuda(table, ids)
    assert ids.dtype == torch.int32 and table.is_contiguous()
    N, W = ids.shape[0], table.shape[1]
    x = torch.empty(N, W, device=ids.device, dtype=torch.float32)
    xb = x if table.dtype == torch.float32 else torch.empty(N, W, device=ids.device, dtype=table.dtype)
    rc = _lib_dec().b200dec_embed(table.data_ptr(), _elem(table.dtype), ids.data_ptr(), x.data_ptr(), None if xb is x else xb.data_ptr(),
                                  N, W, table.shape[0], K.status_word(ids.device).data_ptr(), K._stream())
    _lib.check(rc, "embed")
    return x, xb


@K._ranged
def scaled_add_norm(x: torch.Tensor, delta: torch.Tensor | None, weight: torch.Tensor, alpha: float, eps: float, dtype: torch.dtype,
                    index: torch.Tensor | None = None, keep: bool = True, zero: torch.Tensor | None = None):
    """y = rmsnorm(alpha * x + delta) * weight, all in 32-bit; (y fp32 written over x, y in `dtype`).  `index` int32
    [rows, top]: delta is the sum of those rows of it.  keep = False: only the copy in `dtype` is made.  `zero`: an
    int32 tensor cleared on the way."""
    K._require_cuda(x, weight)
    assert x.dtype == torch.float32 and x.is_contiguous() and weight.dtype == torch.float32
    assert delta is None or (delta.is_contiguous() and delta.dtype == dtype)
    N, W = x.shape
    xb = None
    if dtype != torch.float32 or not keep:
        xb = torch.empty(N, W, device=x.device, dtype=dtype)
    rc = _lib_dec().b200dec_scaled_add_norm(
        x.data_ptr(), _ptr(delta), _ptr(index), 1 if index is None else index.shape[1], _elem(dtype), weight.data_ptr(), float(alpha),
        float(eps), x.data_ptr() if keep else None, _ptr(xb), N, W, _ptr(zero), 0 if zero is None else zero.numel(), K._stream())
    _lib.check(rc, "scaled_add_norm")
    return x, (x if xb is None else xb)


@K._ranged
def norm_add(x: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, mult: float, eps: float, dtype: torch.dtype) -> torch.Tensor:
    """x += mult * rmsnorm(y) * weight in 32-bit, in place; returns the new rows in `dtype` (x itself when that is fp32)."""
    K._require_cuda(x, y, weight)
    assert x.dtype == weight.dtype == torch.float32 and x.is_contiguous() and y.is_contiguous() and y.shape == x.shape and y.dtype == dtype
    xb = x if dtype == torch.float32 else torch.empty_like(x, dtype=dtype)
    rc = _lib_dec().b200dec_norm_add(x.data_ptr(), y.data_ptr(), _elem(dtype), weight.data_ptr(), float(mult), float(eps),
                                     None if xb is x else xb.data_ptr(), x.shape[0], x.shape[1], K._stream())
    _lib.check(rc, "norm_add")
    return xb


@K._ranged
def silu_mul(gate_up: torch.Tensor, ff: int) -> torch.Tensor:
    """silu(gate) * up of rows gate [ff] | up [ff]."""
    K._require_cuda(gate_up)
    assert gate_up.stride(1) == 1 and gate_up.shape[1] >= 2 * ff
    out = torch.empty(gate_up.shape[0], ff, device=gate_up.device, dtype=gate_up.dtype)
    rc = _lib_dec().b200dec_silu_mul(gate_up.data_ptr(), gate_up.stride(0), gate_up.element_size(), out.data_ptr(), ff, gate_up.shape[0], ff,
                                     K._stream())
    _lib.check(rc, "silu_mul")
    return out


# ----------------------------------------------------------------------------- attention
@K._ranged
def rope_write(qkv: torch.Tensor, rows: Rows, cache: PagedKV, cos_sin: torch.Tensor | None, heads: int, write_kv: bool, unit_norm: bool,
               eps: float) -> torch.Tensor:
    """Rotated (and, with unit_norm, unit root-mean-square) queries [N, heads, round8(k_dim)]; keys and values of the
    rows are written to the cache unless write_kv is False (the layer then attends another layer's cache)."""
    K._require_cuda(qkv, cache.k)
    assert qkv.dtype == cache.k.dtype and qkv.stride(1) == 1
    assert qkv.shape[1] == heads * cache.k_dim + (cache.kv_heads * (cache.k_dim + cache.v_dim) if write_kv else 0)
    q = torch.empty(rows.num_rows, heads, cache.k.shape[3], device=qkv.device, dtype=qkv.dtype)
    cs, ts, rs = cache.struct(), K._table_struct(rows.block_table), rows.struct()
    rc = _lib_dec().b200dec_rope_write(
        qkv.data_ptr(), qkv.stride(0), ctypes.byref(rs), ctypes.byref(cs), ctypes.byref(ts), _ptr(cos_sin),
        0 if cos_sin is None else cos_sin.shape[0], 0 if cos_sin is None else cos_sin.shape[1], heads, int(write_kv), int(unit_norm),
        float(eps), q.data_ptr(), K.status_word(qkv.device).data_ptr(), K._stream())
    _lib.check(rc, "rope_write")
    return q


@K._ranged
def norm_rope_write(qkv: torch.Tensor, rows: Rows, cache: PagedKV, q_norm: torch.Tensor, k_norm: torch.Tensor, eps: float,
                    cos_sin: torch.Tensor | None, heads: int) -> torch.Tensor:
    """As rope_write with the RMS norm over the whole query projection and the whole key projection (weights fp32), before
    a rotation that pairs channels 2i and 2i + 1."""
    K._require_cuda(qkv, cache.k, q_norm, k_norm)
    assert qkv.dtype == cache.k.dtype and qkv.stride(1) == 1 and q_norm.dtype == k_norm.dtype == torch.float32
    assert qkv.shape[1] == heads * cache.k_dim + cache.kv_heads * (cache.k_dim + cache.v_dim)
    assert q_norm.numel() == heads * cache.k_dim and k_norm.numel() == cache.kv_heads * cache.k_dim
    q = torch.empty(rows.num_rows, heads, cache.k.shape[3], device=qkv.device, dtype=qkv.dtype)
    cs, ts, rs = cache.struct(), K._table_struct(rows.block_table), rows.struct()
    rc = _lib_dec().b200dec_norm_rope_write(
        qkv.data_ptr(), qkv.stride(0), ctypes.byref(rs), ctypes.byref(cs), ctypes.byref(ts), q_norm.data_ptr(), k_norm.data_ptr(), float(eps),
        _ptr(cos_sin), 0 if cos_sin is None else cos_sin.shape[0], 0 if cos_sin is None else cos_sin.shape[1], heads, q.data_ptr(),
        K.status_word(qkv.device).data_ptr(), K._stream())
    _lib.check(rc, "norm_rope_write")
    return q


@dataclass
class AttnOptions:
    """window: a row sees itself and the window - 1 tokens before it (0: all).  sink fp32 [heads]: exp(sink) joins the
    softmax denominator.  gate [rows, heads] in the model's precision: head outputs times sigmoid(gate).  out_scale
    multiplies the result."""

    window: int = 0
    sink: torch.Tensor | None = None
    gate: torch.Tensor | None = None
    out_scale: float = 1.0

    def struct(self, out: torch.Tensor) -> _lib.AttnOptions:
        assert self.sink is None or (self.sink.dtype == torch.float32 and self.sink.is_contiguous())
        assert self.gate is None or (self.gate.stride(1) == 1 and self.gate.dtype == out.dtype)
        return _lib.AttnOptions(self.window, _ptr(self.sink), _ptr(self.gate), 0 if self.gate is None else self.gate.stride(0),
                                self.out_scale, out.stride(0))


def _opt(opt: AttnOptions | None, out: torch.Tensor):
    """The option argument of an attention call; `out` [rows, heads, v_dim] may be a part of wider rows with options only."""
    assert out.stride(2) == 1 and out.stride(1) == out.shape[2]
    if opt is None and out.is_contiguous():
        return None
    st = (opt or AttnOptions()).struct(out)
    if out.is_contiguous():
        st.out_stride = 0
    return ctypes.byref(st)


def tensor_core_attention(cache: PagedKV) -> bool:
    return cache.k.dtype == torch.bfloat16 and max(cache.k_dim, cache.v_dim) <= MAX_TENSOR_CORE_DIM and cache.page_size % 16 == 0


@K._ranged
def attention_rows(q: torch.Tensor, cache: PagedKV, rows: Rows, scale: float, opt: AttnOptions | None = None,
                   out: torch.Tensor | None = None) -> torch.Tensor:
    """Causal attention of every row over the cache on the CUDA cores, 32-bit: any sizes, both precisions."""
    K._require_cuda(q, cache.k)
    if out is None:
        out = torch.empty(q.shape[0], q.shape[1], cache.v_dim, device=q.device, dtype=q.dtype)
    cs, ts, rs = cache.struct(), K._table_struct(rows.block_table), rows.struct()
    rc = _lib_dec().b200dec_attn_rows_opt(q.data_ptr(), ctypes.byref(cs), ctypes.byref(ts), ctypes.byref(rs), q.shape[1], float(scale),
                                          _opt(opt, out), out.data_ptr(), K.status_word(q.device).data_ptr(), K._stream())
    _lib.check(rc, "attention_rows")
    return out


@K._ranged
def paged_decode_attention(q: torch.Tensor, cache: PagedKV, rows: Rows, scale: float, out: torch.Tensor, zero_idle: bool,
                           opt: AttnOptions | None = None) -> None:
    """The decoding entries' rows (the first ones of q and out) on the tensor cores."""
    K._require_cuda(q, cache.k)
    lib, dev, sms = _lib_dec(), q.device, K.num_sms(q.device)
    B, heads = rows.cached_lens.shape[0], q.shape[1]
    nbytes = lib.b200dec_decode_attn_workspace(B, heads, cache.kv_heads, cache.v_dim, sms)
    ws = K.decode_workspace(dev, ("paged", B, cache.v_dim), heads, cache.kv_heads, nbytes)
    cs, ts = cache.struct(), K._table_struct(rows.block_table)
    rc = lib.b200dec_decode_attn_opt(q.data_ptr(), ctypes.byref(cs), ctypes.byref(ts), K._i32(rows.cached_lens), K._i32(rows.num_decoding),
                                     B, heads, float(scale), _opt(opt, out), out.data_ptr(), int(zero_idle), ws.data_ptr(), ws.numel(), sms,
                                     K.status_word(dev).data_ptr(), K._stream())
    _lib.check(rc, "paged_decode_attention")


@K._ranged
def paged_prefill_attention(q: torch.Tensor, cache: PagedKV, rows: Rows, scale: float, out: torch.Tensor,
                            opt: AttnOptions | None = None) -> None:
    """The prompt portions' rows on tcgen05, keys and values by page from the cache."""
    K._require_cuda(q, cache.k)
    cs, ts = cache.struct(), K._table_struct(rows.block_table)
    rc = _lib_dec().b200dec_prefill_attn_opt(
        q.data_ptr(), ctypes.byref(cs), ctypes.byref(ts), K._i32(rows.seq_ids), K._i32(rows.cu_seqlens), K._i32(rows.cached_lens),
        K._i32(rows.tile_start), rows.tile_start.shape[0], rows.block_m, rows.num_rows, q.shape[1], float(scale), _opt(opt, out),
        out.data_ptr(), K.status_word(q.device).data_ptr(), K._stream())
    _lib.check(rc, "paged_prefill_attention")


def paged_attention(q: torch.Tensor, cache: PagedKV, rows: Rows, scale: float, opt: AttnOptions | None = None,
                    out: torch.Tensor | None = None) -> torch.Tensor:
    """Attention of a step's rows over the paged cache: [N, heads, v_dim] (written to `out` if given)."""
    if not tensor_core_attention(cache):
        return attention_rows(q, cache, rows, scale, opt, out)
    if out is None:
        out = torch.empty(q.shape[0], q.shape[1], cache.v_dim, device=q.device, dtype=q.dtype)
    if rows.seq_ids is not None:
        paged_prefill_attention(q, cache, rows, scale, out, opt)
    paged_decode_attention(q, cache, rows, scale, out, rows.seq_ids is None, opt)
    return out


# ----------------------------------------------------------------------------- mixture of experts
@dataclass
class Experts:
    """Weights of one layer's experts: gate and up rows interleaved (row 2f = gate f, row 2f + 1 = up f), so that one
    product yields both inputs of an output channel side by side."""

    router: torch.Tensor  # bf16 [experts, width]
    gate_up: torch.Tensor  # [experts, 2 * ff, width]
    down: torch.Tensor  # [experts, width, ff]
    top: int
    limit: float
    slope: float
    counts: torch.Tensor  # int32 [experts], zero before every use

    @property
    def num(self) -> int:
        return self.gate_up.shape[0]


def make_experts(router, gates, ups, downs, top: int, limit: float, slope: float, dtype, device) -> Experts:
    """Interleave and stack per-expert gate / up [ff, width] and down [width, ff] matrices."""
    E, (F, W) = len(gates), gates[0].shape
    gate_up = torch.empty(E, F, 2, W, dtype=dtype, device=device)
    down = torch.empty(E, W, F, dtype=dtype, device=device)
    for e in range(E):
        gate_up[e, :, 0] = gates[e].to(device, dtype)
        gate_up[e, :, 1] = ups[e].to(device, dtype)
        down[e] = downs[e].to(device, dtype)
    return Experts(router.to(device, torch.bfloat16).contiguous(), gate_up.view(E, 2 * F, W), down, top, limit, slope,
                   torch.zeros(E, dtype=torch.int32, device=device))


def expert_tile_rows(num_rows: int, top: int, experts: int, dtype) -> int:
    """Most rows of an expert's tile: 256 for prompt-sized steps (the widest tcgen05 tile), 64 for small ones, where
    weights are streamed and a narrow tile leaves shared memory for a deeper ring."""
    if dtype == torch.float32:
        return 32
    total = num_rows * top
    return 64 if total <= 512 or total <= 48 * experts else 256


def max_expert_tiles(total: int, experts: int, tile_rows: int) -> int:
    return total // tile_rows + min(experts, total)


def grouped_linear(x, w, tiles, max_tiles, tile_rows, scores=None, limit=0.0, slope=0.0, variant: int | None = None):
    """Rows of x (ordered by expert) times their expert's matrix w [E, out, in]; with scores: the gated unit, half as
    many outputs."""
    rows, width = x.shape
    E, out_rows, _ = w.shape
    act = scores is not None
    if variant is None:
        variant = 0 if x.dtype == torch.bfloat16 and width % 8 == 0 else 1
    y = torch.empty(rows, out_rows // 2 if act else out_rows, device=x.device, dtype=x.dtype)
    rc = _lib_dec().b200dec_grouped_linear(
        x.data_ptr(), w.data_ptr(), x.element_size(), tiles.data_ptr(), max_tiles, tile_rows, rows, E, out_rows, width, _ptr(scores),
        int(act), float(limit), float(slope), y.data_ptr(), K.num_sms(x.device), variant, K.status_word(x.device).data_ptr(), K._stream())
    _lib.check(rc, "grouped_linear")
    return y


@K._ranged
def mixture(x: torch.Tensor, xb: torch.Tensor, ex: Experts, variant: int | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """Routed experts of every row.  x: the rows in fp32 (the router's input), xb: in the model's precision.  The score
    multiplies the expert's input.  Returns (outputs [N * top, width] ordered by expert, places int32 [N, top]): the
    layer's output for row r is the sum of outputs[places[r]] (scaled_add_norm takes both).  `ex.counts` must be
    zero, which scaled_add_norm(zero=ex.counts) sees to."""
    K._require_cuda(x, xb, ex.gate_up)
    lib, dev = _lib_dec(), x.device
    N, W = x.shape
    total, E = N * ex.top, ex.num
    tile_rows = expert_tile_rows(N, ex.top, E, xb.dtype)
    max_tiles = max_expert_tiles(total, E, tile_rows)
    # separate allocations: no kernel of the chain reads a cache line that the next one's input shares
    ids, ranks, slots, scores = (torch.empty(total, dtype=torch.int32, device=dev) for _ in range(4))
    tiles = torch.empty(1 + 3 * max_tiles, dtype=torch.int32, device=dev)
    score_sorted = torch.empty(total, dtype=torch.float32, device=dev)
    rc = lib.b200dec_router(x.data_ptr(), ex.router.data_ptr(), N, W, E, ex.top, ids.data_ptr(), scores.data_ptr(), ranks.data_ptr(),
                            ex.counts.data_ptr(), K._stream())
    _lib.check(rc, "router")
    xs = torch.empty(total, W, device=dev, dtype=xb.dtype)
    rc = lib.b200dec_dispatch(xb.data_ptr(), xb.element_size(), ids.data_ptr(), scores.data_ptr(), ranks.data_ptr(), ex.counts.data_ptr(), N,
                              W, E, ex.top, tile_rows, xs.data_ptr(), score_sorted.data_ptr(), slots.data_ptr(), tiles.data_ptr(), max_tiles,
                              K._stream())
    _lib.check(rc, "dispatch")
    h = grouped_linear(xs, ex.gate_up, tiles, max_tiles, tile_rows, score_sorted, ex.limit, ex.slope, variant)
    return grouped_linear(h, ex.down, tiles, max_tiles, tile_rows, variant=variant), slots.view(N, ex.top)


# ----------------------------------------------------------------------------- recurrent layers
@dataclass
class Recurrence:
    """Constants of a layer that carries a state S [dim, vdim] per head (include/b200dec.h, b200dec_recurrence):
    S <- decay S; u = beta (v - S^T k) with `correct`, else step * v; S <- S + k u^T; o = S^T q + skip v."""

    heads: int
    qk_heads: int
    dim: int
    vdim: int
    conv_w: torch.Tensor  # fp32 [taps, channels], last row: the current token
    conv_b: torch.Tensor | None  # fp32 [channels]
    neg_a: torch.Tensor  # fp32 [heads]: decay = exp(neg_a * softplus(step_in + dt_bias))
    dt_bias: torch.Tensor  # fp32 [heads], or [heads * dim] with channel_decay
    skip: torch.Tensor | None  # fp32 [heads]
    off_q: int
    off_k: int
    off_v: int
    channel_decay: bool = False
    correct: bool = False
    unit_eps: float | None = None  # unit q and k per head, x / sqrt(sum(x^2) + unit_eps)
    q_scale: float = 1.0

    @property
    def taps(self) -> int:
        return self.conv_w.shape[0]

    @property
    def channels(self) -> int:
        return self.conv_w.shape[1]


@dataclass
class RecurrentState:
    """What a recurrent layer keeps per request slot: the 32-bit state and the convolution's last raw inputs by position."""

    state: torch.Tensor  # fp32 [slots, heads, dim, round4(vdim)]
    ring: torch.Tensor  # [slots, taps, channels]


def make_recurrent_state(rec: Recurrence, slots: int, dtype, device) -> RecurrentState:
    return RecurrentState(torch.zeros(slots, rec.heads, rec.dim, (rec.vdim + 3) // 4 * 4, device=device),
                          torch.zeros(slots, rec.taps, rec.channels, dtype=dtype, device=device))


@dataclass
class GatedNorm:
    """Norm of a row's `parts` equal parts by themselves: times silu(gate) before (gate_first) or sigmoid(gate) after."""

    weight: torch.Tensor  # fp32, repeated along the row
    parts: int
    eps: float
    gate_first: bool
    out_scale: float = 1.0


def _recurrence_args(rec: Recurrence, st: RecurrentState, x, step, beta):
    assert x.stride(1) == 1 and x.shape[1] == rec.channels and x.dtype == st.ring.dtype and step.stride(1) == 1 and step.dtype == x.dtype
    assert st.state.is_contiguous() and st.ring.is_contiguous() and (beta is None or (beta.stride(1) == 1 and beta.dtype == x.dtype))
    assert step.shape[1] == rec.heads * (rec.dim if rec.channel_decay else 1) == rec.dt_bias.numel()
    r = _lib.Recurrence(st.state.data_ptr(), st.ring.data_ptr(), rec.conv_w.data_ptr(), _ptr(rec.conv_b), rec.neg_a.data_ptr(),
                        rec.dt_bias.data_ptr(), _ptr(rec.skip), st.state.shape[0], rec.heads, rec.qk_heads, rec.dim, rec.vdim, rec.taps,
                        x.element_size(), rec.channels, rec.off_q, rec.off_k, rec.off_v, int(rec.channel_decay), int(rec.correct),
                        int(rec.unit_eps is not None), rec.unit_eps or 0.0, rec.q_scale)
    i = _lib.RecurrenceIn(x.data_ptr(), step.data_ptr(), _ptr(beta), x.stride(0), step.stride(0), 0 if beta is None else beta.stride(0))
    return r, i


@K._ranged
def recurrence_decode(rec: Recurrence, st: RecurrentState, x, step, beta, rows: Rows, out: torch.Tensor, norm: GatedNorm | None = None,
                      gate: torch.Tensor | None = None, variant: int = 0) -> None:
    """One token of every decoding entry: convolution, state and read-out; out fp32 [N, heads * vdim], or with `norm` (one part
    per head, gate behind it) the gated output in the model's precision."""
    K._require_cuda(x, out, st.state)
    r, i = _recurrence_args(rec, st, x, step, beta)
    e = rows.entries()
    rc = _lib_dec().b200dec_recurrence_decode(
        ctypes.byref(r), ctypes.byref(i), ctypes.byref(e), None if norm is None else norm.weight.data_ptr(), 0.0 if norm is None else norm.eps,
        _ptr(gate), 0 if gate is None else gate.stride(0), out.data_ptr(), out.stride(0), variant, K.num_sms(x.device),
        K.status_word(x.device).data_ptr(), K._stream())
    _lib.check(rc, "recurrence_decode")


@K._ranged
def conv_rows(rec: Recurrence, st: RecurrentState, x, step, beta, rows: Rows) -> torch.Tensor:
    """silu(convolution) of the prompt portions' rows, all channels."""
    K._require_cuda(x, st.ring)
    r, i = _recurrence_args(rec, st, x, step, beta)
    e = rows.entries()
    conv = torch.empty(rows.num_rows, _round8(rec.channels), device=x.device, dtype=x.dtype)
    rc = _lib_dec().b200dec_conv_rows(ctypes.byref(r), ctypes.byref(i), ctypes.byref(e), conv.data_ptr(), K.status_word(x.device).data_ptr(),
                                      K._stream())
    _lib.check(rc, "conv_rows")
    return conv


@K._ranged
def recurrence_prefill(rec: Recurrence, st: RecurrentState, x, step, beta, rows: Rows, out: torch.Tensor, form: str | None = None) -> None:
    """The prompt portions' rows: convolution, then the state through every portion; out fp32 [N, heads * vdim].  `form`: which
    kernel carries the state ("scan" token by token, any sizes; "blocked", "chunked"); default: the fastest that applies."""
    K._require_cuda(x, out, st.state)
    conv = conv_rows(rec, st, x, step, beta, rows)
    r, i = _recurrence_args(rec, st, x, step, beta)
    e = rows.entries()
    lib, status = _lib_dec(), K.status_word(x.device).data_ptr()
    sizes = {"chunked": lib.b200dec_state_space_chunked_workspace(ctypes.byref(r)),
             "blocked": lib.b200dec_recurrence_blocked_workspace(ctypes.byref(r), ctypes.byref(e)) if rec.skip is None else 0}
    if form is None:
        form = next((f for f, n in sizes.items() if n), "scan")
    if form == "scan":
        rc = lib.b200dec_recurrence_scan(ctypes.byref(r), ctypes.byref(i), conv.data_ptr(), ctypes.byref(e), out.data_ptr(), status, K._stream())
    else:
        ws = torch.empty(sizes[form], dtype=torch.uint8, device=x.device)
        args = (ctypes.byref(r), ctypes.byref(i), conv.data_ptr(), ctypes.byref(e), out.data_ptr(), ws.data_ptr(), sizes[form])
        if form == "chunked":
            rc = lib.b200dec_state_space_chunked(*args, K.num_sms(x.device), status, K._stream())
        else:
            rc = lib.b200dec_recurrence_blocked(*args, status, K._stream())
    _lib.check(rc, f"recurrence_{form}")


@K._ranged
def gated_norm(o: torch.Tensor, gate: torch.Tensor, norm: GatedNorm, out: torch.Tensor) -> None:
    K._require_cuda(o, gate, out)
    assert o.is_contiguous() and o.dtype == torch.float32 and gate.stride(1) == 1 and gate.dtype == out.dtype and out.stride(1) == 1
    assert gate.shape == o.shape == out.shape and norm.weight.dtype == torch.float32
    rc = _lib_dec().b200dec_gated_norm(o.data_ptr(), gate.data_ptr(), gate.stride(0), int(norm.gate_first), out.element_size(),
                                       norm.weight.data_ptr(), norm.weight.numel(), norm.eps, norm.out_scale, out.data_ptr(), out.stride(0),
                                       o.shape[0], o.shape[1], norm.parts, K._stream())
    _lib.check(rc, "gated_norm")


def recurrent_mixer(rec: Recurrence, st: RecurrentState, x, step, beta, gate, norm: GatedNorm, rows: Rows, out: torch.Tensor) -> None:
    """A recurrent layer between its projections: out [N, heads * vdim] in the model's precision."""
    if rows.seq_ids is None and not norm.gate_first and norm.parts == rec.heads and norm.weight.numel() == rec.vdim and norm.out_scale == 1.0:
        return recurrence_decode(rec, st, x, step, beta, rows, out, norm, gate)
    o = torch.empty(x.shape[0], rec.heads * rec.vdim, device=x.device, dtype=torch.float32)
    recurrence_decode(rec, st, x, step, beta, rows, o)
    if rows.seq_ids is not None:
        recurrence_prefill(rec, st, x, step, beta, rows, o)
    gated_norm(o, gate, norm, out)


# ----------------------------------------------------------------------------- projections side by side
class Packed:
    """Matrices with a common input as one product.  Every part starts at a multiple of 8 output channels, so that the parts
    of a row can be read in vectors."""

    def __init__(self, parts: dict[str, torch.Tensor], dtype, device):
        self.at: dict[str, tuple[int, int]] = {}
        blocks, n = [], 0
        for name, w in parts.items():
            self.at[name] = (n, n + w.shape[0])
            pad = -w.shape[0] % 8
            blocks.append(w.to(device, dtype))
            if pad:
                blocks.append(torch.zeros(pad, w.shape[1], dtype=dtype, device=device))
            n += w.shape[0] + pad
        self.weight = torch.cat(blocks)

    def __call__(self, x: torch.Tensor) -> torch.Tensor:
        return K.linear(x, self.weight)

    def part(self, y: torch.Tensor, name: str) -> torch.Tensor:
        lo, hi = self.at[name]
        return y[:, lo:hi]
