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

    def struct(self) -> _lib.DecRows:
        return _lib.DecRows(_ptr(self.seq_ids), _ptr(self.positions), K._i32(self.cached_lens), K._i32(self.num_decoding),
                            self.num_rows)


# ----------------------------------------------------------------------------- rotary positions
@dataclass(frozen=True)
class Rotary:
    """Rotation of the first `dims` channels of a head, channel i paired with i + dims / 2.  With `scaling` (factor,
    original, fast, slow) the frequencies are stretched as YaRN does (Peng et al., "YaRN: Efficient Context Window
    Extension of Large Language Models"): components that turn more than `fast` times within the original context
    keep their frequency, those that turn less than `slow` times are divided by `factor`, a linear ramp joins the two,
    and cos and sin are multiplied by 0.1 ln(factor) + 1."""

    dims: int
    base: float
    scaling: tuple[float, float, float, float] | None = None  # factor, original, fast, slow

    def frequencies(self) -> tuple[list[float], float]:
        half = self.dims // 2
        freq = [self.base ** (-2.0 * i / self.dims) for i in range(half)]
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


def tensor_core_attention(cache: PagedKV) -> bool:
    return cache.k.dtype == torch.bfloat16 and max(cache.k_dim, cache.v_dim) <= MAX_TENSOR_CORE_DIM and cache.page_size % 16 == 0


@K._ranged
def attention_rows(q: torch.Tensor, cache: PagedKV, rows: Rows, scale: float) -> torch.Tensor:
    """Causal attention of every row over the cache on the CUDA cores, 32-bit: any sizes, both precisions."""
    K._require_cuda(q, cache.k)
    out = torch.empty(q.shape[0], q.shape[1], cache.v_dim, device=q.device, dtype=q.dtype)
    cs, ts, rs = cache.struct(), K._table_struct(rows.block_table), rows.struct()
    rc = _lib_dec().b200dec_attn_rows(q.data_ptr(), ctypes.byref(cs), ctypes.byref(ts), ctypes.byref(rs), q.shape[1], float(scale),
                                      out.data_ptr(), K.status_word(q.device).data_ptr(), K._stream())
    _lib.check(rc, "attention_rows")
    return out


@K._ranged
def paged_decode_attention(q: torch.Tensor, cache: PagedKV, rows: Rows, scale: float, out: torch.Tensor, zero_idle: bool) -> None:
    """The decoding entries' rows (the first ones of q and out) on the tensor cores."""
    K._require_cuda(q, cache.k)
    lib, dev, sms = _lib_dec(), q.device, K.num_sms(q.device)
    B, heads = rows.cached_lens.shape[0], q.shape[1]
    nbytes = lib.b200dec_decode_attn_workspace(B, heads, cache.kv_heads, cache.v_dim, sms)
    ws = K.decode_workspace(dev, ("paged", B, cache.v_dim), heads, cache.kv_heads, nbytes)
    cs, ts = cache.struct(), K._table_struct(rows.block_table)
    rc = lib.b200dec_decode_attn(q.data_ptr(), ctypes.byref(cs), ctypes.byref(ts), K._i32(rows.cached_lens), K._i32(rows.num_decoding), B,
                                 heads, float(scale), out.data_ptr(), int(zero_idle), ws.data_ptr(), ws.numel(), sms,
                                 K.status_word(dev).data_ptr(), K._stream())
    _lib.check(rc, "paged_decode_attention")


@K._ranged
def paged_prefill_attention(q: torch.Tensor, cache: PagedKV, rows: Rows, scale: float, out: torch.Tensor) -> None:
    """The prompt portions' rows on tcgen05, keys and values by page from the cache."""
    K._require_cuda(q, cache.k)
    cs, ts = cache.struct(), K._table_struct(rows.block_table)
    rc = _lib_dec().b200dec_prefill_attn(
        q.data_ptr(), ctypes.byref(cs), ctypes.byref(ts), K._i32(rows.seq_ids), K._i32(rows.cu_seqlens), K._i32(rows.cached_lens),
        K._i32(rows.tile_start), rows.tile_start.shape[0], rows.block_m, rows.num_rows, q.shape[1], float(scale), out.data_ptr(),
        K.status_word(q.device).data_ptr(), K._stream())
    _lib.check(rc, "paged_prefill_attention")


def paged_attention(q: torch.Tensor, cache: PagedKV, rows: Rows, scale: float) -> torch.Tensor:
    """Attention of a step's rows over the paged cache: [N, heads, v_dim]."""
    if not tensor_core_attention(cache):
        return attention_rows(q, cache, rows, scale)
    out = torch.empty(q.shape[0], q.shape[1], cache.v_dim, device=q.device, dtype=q.dtype)
    if rows.seq_ids is not None:
        paged_prefill_attention(q, cache, rows, scale, out)
    paged_decode_attention(q, cache, rows, scale, out, zero_idle=rows.seq_ids is None)
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
