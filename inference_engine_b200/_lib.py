"""ctypes binding of libb200kv.so (include/b200kv.h) and libb200dec.so (include/b200dec.h).

Loading never falls back to anything: a missing or unloadable library raises, and every
wrapper raises on a negative return code."""
from __future__ import annotations

import ctypes as C
import os

from . import build as _build

c_void_p, c_int32, c_int64, c_float, c_size_t = C.c_void_p, C.c_int32, C.c_int64, C.c_float, C.c_size_t


class Cache(C.Structure):
    """struct b200kv_cache"""

    _fields_ = [
        ("k", c_void_p), ("v", c_void_p), ("k_scale", c_void_p), ("v_scale", c_void_p), ("k_calibration", c_void_p),
        ("stride_page", c_int64), ("stride_head", c_int64), ("stride_tok", c_int64),
        ("sstride_page", c_int64), ("sstride_head", c_int64),
        ("cstride_page", c_int64), ("cstride_head", c_int64),
        ("num_pages", c_int32), ("num_kv_heads", c_int32), ("page_size", c_int32), ("head_dim", c_int32),
    ]


class Table(C.Structure):
    """struct b200kv_table"""

    _fields_ = [("ids", c_void_p), ("stride", c_int32), ("max_pages", c_int32)]


class DecCache(C.Structure):
    """struct b200dec_cache"""

    _fields_ = [("k", c_void_p), ("v", c_void_p), ("num_pages", c_int32), ("kv_heads", c_int32), ("page_size", c_int32),
                ("k_dim", c_int32), ("v_dim", c_int32), ("k_row", c_int32), ("v_row", c_int32), ("elem", c_int32)]


class DecRows(C.Structure):
    """struct b200dec_rows"""

    _fields_ = [("seq_ids", c_void_p), ("positions", c_void_p), ("cached_lens", c_void_p), ("num_decoding", c_void_p),
                ("num_rows", c_int32)]


class AttnOptions(C.Structure):
    """struct b200dec_attn_options"""

    _fields_ = [("window", c_int32), ("sink", c_void_p), ("gate", c_void_p), ("gate_stride", c_int64), ("out_scale", c_float),
                ("out_stride", c_int64)]


class Recurrence(C.Structure):
    """struct b200dec_recurrence"""

    _fields_ = [(n, c_void_p) for n in ("state", "ring", "conv_w", "conv_b", "neg_a", "dt_bias", "skip")] + [
        (n, c_int32) for n in ("num_slots", "heads", "qk_heads", "dim", "vdim", "taps", "elem", "channels", "off_q", "off_k", "off_v",
                               "channel_decay", "correct", "unit_norm")] + [("unit_eps", c_float), ("q_scale", c_float)]


class RecurrenceIn(C.Structure):
    """struct b200dec_recurrence_in"""

    _fields_ = [("x", c_void_p), ("step", c_void_p), ("beta", c_void_p), ("x_stride", c_int64), ("step_stride", c_int64),
                ("beta_stride", c_int64)]


class Entries(C.Structure):
    """struct b200dec_entries"""

    _fields_ = [(n, c_void_p) for n in ("cu_seqlens", "cached_lens", "num_decoding", "slots", "seq_ids", "positions")] + [
        ("num_entries", c_int32), ("num_rows", c_int32)]


P_CACHE, P_TABLE = C.POINTER(Cache), C.POINTER(Table)
P_DCACHE, P_ROWS, P_OPT = C.POINTER(DecCache), C.POINTER(DecRows), C.POINTER(AttnOptions)
P_REC, P_REC_IN, P_ENT = C.POINTER(Recurrence), C.POINTER(RecurrenceIn), C.POINTER(Entries)

# name -> (restype, argtypes); must list every function include/b200kv.h declares
SIGNATURES = {
    "b200kv_version": (c_int32, []),
    "b200kv_error_string": (C.c_char_p, [c_int32]),
    "b200kv_write_decode": (c_int32, [c_void_p, c_int64, c_int64, c_void_p, c_int64, c_int64, c_void_p, c_int64, c_int64,
                                      c_void_p, c_void_p, c_void_p, c_int64, c_void_p, c_int64, P_CACHE, P_TABLE,
                                      c_void_p, c_void_p, c_void_p, c_int64, c_int64, c_int32, c_int32, c_float,
                                      c_void_p, c_void_p]),
    "b200kv_norm_rope_prefill": (c_int32, [c_void_p, c_int64, c_int64, c_void_p, c_int64, c_int64, c_void_p, c_void_p,
                                           c_void_p, c_int64, c_void_p, c_int64, c_void_p, c_int64, c_int64, c_void_p,
                                           c_int64, c_int64, c_int32, c_int32, c_int32, c_int32, c_float, c_void_p]),
    "b200kv_quantize_prefill": (c_int32, [c_void_p, c_int64, c_int64, c_void_p, c_int64, c_int64, c_void_p, c_int32,
                                          P_CACHE, P_TABLE, c_void_p, c_void_p, c_int32, c_void_p, c_void_p]),
    "b200kv_write_prefill": (c_int32, [c_void_p, c_int64, c_int64, c_void_p, c_int64, c_int64, c_void_p, c_int64, c_int64,
                                       c_void_p, c_void_p, c_void_p, c_int64, c_void_p, c_int64, c_void_p, c_int32,
                                       P_CACHE, P_TABLE, c_void_p, c_void_p, c_void_p, c_int64, c_int64, c_void_p, c_int64,
                                       c_int64, c_int32, c_int32, c_float, c_void_p, c_void_p]),
    "b200kv_dequant_prefix": (c_int32, [P_CACHE, P_TABLE, c_void_p, c_int32, c_void_p, c_void_p, c_int64, c_int64,
                                        c_int32, c_void_p, c_void_p]),
    "b200kv_prefill_attn": (c_int32, [c_void_p, c_int64, c_int64, c_void_p, c_int64, c_int64, c_void_p, c_int64, c_int64,
                                      c_void_p, c_void_p, c_void_p, c_int32, c_int32, c_void_p, c_void_p, c_int64,
                                      c_int64, c_void_p, c_void_p, c_int64, c_int64, c_int32, c_int32, c_int32, c_int32,
                                      c_void_p]),
    "b200kv_prefill_attn_variant": (c_int32, [c_void_p, c_int64, c_int64, c_void_p, c_int64, c_int64, c_void_p, c_int64,
                                              c_int64, c_void_p, c_void_p, c_void_p, c_int32, c_int32, c_void_p, c_void_p,
                                              c_int64, c_int64, c_int32, c_void_p, c_void_p, c_int64, c_int64, c_int32,
                                              c_int32, c_int32, c_int32, c_int32, c_void_p, c_void_p]),
    "b200kv_silu_mul": (c_int32, [c_void_p, c_int64, c_void_p, c_int64, c_int32, c_int32, c_void_p]),
    "b200kv_add_rms_norm": (c_int32, [c_void_p, c_int64, c_void_p, c_int64, c_void_p, c_void_p, c_int64, c_void_p, c_int64,
                                      c_int32, c_int32, c_float, c_void_p]),
    "b200kv_sample_workspace_bytes": (c_size_t, [c_int32, c_int32]),
    "b200kv_sample": (c_int32, [c_void_p, c_int64, c_int32, c_void_p, c_float, c_void_p, c_size_t, c_void_p, c_int64,
                                c_int32, c_int32, c_void_p]),
    "b200kv_skinny_linear": (c_int32, [c_void_p, c_int64, c_void_p, c_int64, c_void_p, c_int64, c_int32, c_int32, c_int32,
                                       c_int32, c_void_p, c_void_p]),
    "b200kv_set_chained_launch": (None, [c_int32]),
    "b200kv_get_chained_launch": (c_int32, []),
    "b200kv_decode_attn_workspace_bytes": (c_size_t, [c_int32, c_int32, c_int32, c_int32, c_int32]),
    "b200kv_decode_attn_workspace_zero_bytes": (c_size_t, [c_int32, c_int32]),
    "b200kv_decode_attn": (c_int32, [c_void_p, c_int64, c_int64, P_CACHE, P_TABLE, c_void_p, c_void_p, c_float, c_void_p,
                                     c_int64, c_int64, c_void_p, c_size_t, c_int32, c_int32, c_int32, c_int32, c_void_p,
                                     c_void_p]),
    "b200kv_decode_plan_bytes": (c_size_t, [c_int32]),
    "b200kv_decode_plan": (c_int32, [P_TABLE, c_void_p, c_void_p, c_int32, c_int32, c_int32, c_int32, c_void_p, c_size_t,
                                     c_void_p]),
    "b200kv_decode_attn_planned": (c_int32, [c_void_p, c_int64, c_int64, P_CACHE, P_TABLE, c_void_p, c_void_p, c_float,
                                             c_void_p, c_int64, c_int64, c_void_p, c_size_t, c_void_p, c_size_t, c_int32,
                                             c_int32, c_int32, c_int32, c_void_p, c_void_p]),
    "b200kv_decode_attn_static_limit": (c_size_t, []),
    "b200kv_decode_attn_static": (c_int32, [c_void_p, c_int64, c_int64, P_CACHE, P_TABLE, c_void_p, c_void_p, c_float,
                                            c_void_p, c_int64, c_int64, c_int32, c_int32, c_int32, c_void_p, c_void_p]),
}

# entry points of libb200dec.so: every function include/b200dec.h declares, and the ones it shares with libb200kv.so
DECODER_SIGNATURES = {
    "b200dec_embed": (c_int32, [c_void_p, c_int32, c_void_p, c_void_p, c_void_p, c_int32, c_int32, c_int32, c_void_p, c_void_p]),
    "b200dec_scaled_add_norm": (c_int32, [c_void_p, c_void_p, c_void_p, c_int32, c_int32, c_void_p, c_float, c_float, c_void_p,
                                          c_void_p, c_int32, c_int32, c_void_p, c_int32, c_void_p]),
    "b200dec_rope_write": (c_int32, [c_void_p, c_int64, P_ROWS, P_DCACHE, P_TABLE, c_void_p, c_int32, c_int32, c_int32, c_int32,
                                     c_int32, c_float, c_void_p, c_void_p, c_void_p]),
    "b200dec_attn_rows": (c_int32, [c_void_p, P_DCACHE, P_TABLE, P_ROWS, c_int32, c_float, c_void_p, c_void_p, c_void_p]),
    "b200dec_decode_attn_workspace": (c_size_t, [c_int32, c_int32, c_int32, c_int32, c_int32]),
    "b200dec_decode_attn": (c_int32, [c_void_p, P_DCACHE, P_TABLE, c_void_p, c_void_p, c_int32, c_int32, c_float, c_void_p, c_int32,
                                      c_void_p, c_size_t, c_int32, c_void_p, c_void_p]),
    "b200dec_prefill_attn": (c_int32, [c_void_p, P_DCACHE, P_TABLE, c_void_p, c_void_p, c_void_p, c_void_p, c_int32, c_int32, c_int32,
                                       c_int32, c_float, c_void_p, c_void_p, c_void_p]),
    "b200dec_attn_rows_opt": (c_int32, [c_void_p, P_DCACHE, P_TABLE, P_ROWS, c_int32, c_float, P_OPT, c_void_p, c_void_p, c_void_p]),
    "b200dec_decode_attn_opt": (c_int32, [c_void_p, P_DCACHE, P_TABLE, c_void_p, c_void_p, c_int32, c_int32, c_float, P_OPT, c_void_p,
                                          c_int32, c_void_p, c_size_t, c_int32, c_void_p, c_void_p]),
    "b200dec_prefill_attn_opt": (c_int32, [c_void_p, P_DCACHE, P_TABLE, c_void_p, c_void_p, c_void_p, c_void_p, c_int32, c_int32, c_int32,
                                           c_int32, c_float, P_OPT, c_void_p, c_void_p, c_void_p]),
    "b200dec_norm_rope_write": (c_int32, [c_void_p, c_int64, P_ROWS, P_DCACHE, P_TABLE, c_void_p, c_void_p, c_float, c_void_p, c_int32,
                                          c_int32, c_int32, c_void_p, c_void_p, c_void_p]),
    "b200dec_norm_add": (c_int32, [c_void_p, c_void_p, c_int32, c_void_p, c_float, c_float, c_void_p, c_int32, c_int32, c_void_p]),
    "b200dec_silu_mul": (c_int32, [c_void_p, c_int64, c_int32, c_void_p, c_int64, c_int32, c_int32, c_void_p]),
    "b200dec_recurrence_decode": (c_int32, [P_REC, P_REC_IN, P_ENT, c_void_p, c_float, c_void_p, c_int64, c_void_p, c_int64, c_int32,
                                            c_int32, c_void_p, c_void_p]),
    "b200dec_conv_rows": (c_int32, [P_REC, P_REC_IN, P_ENT, c_void_p, c_void_p, c_void_p]),
    "b200dec_recurrence_scan": (c_int32, [P_REC, P_REC_IN, c_void_p, P_ENT, c_void_p, c_void_p, c_void_p]),
    "b200dec_recurrence_blocked_workspace": (c_size_t, [P_REC, P_ENT]),
    "b200dec_recurrence_blocked": (c_int32, [P_REC, P_REC_IN, c_void_p, P_ENT, c_void_p, c_void_p, c_size_t, c_void_p, c_void_p]),
    "b200dec_state_space_chunked_workspace": (c_size_t, [P_REC]),
    "b200dec_state_space_chunked": (c_int32, [P_REC, P_REC_IN, c_void_p, P_ENT, c_void_p, c_void_p, c_size_t, c_int32, c_void_p, c_void_p]),
    "b200dec_gated_norm": (c_int32, [c_void_p, c_void_p, c_int64, c_int32, c_int32, c_void_p, c_int32, c_float, c_float, c_void_p, c_int64,
                                     c_int32, c_int32, c_int32, c_void_p]),
    "b200dec_router": (c_int32, [c_void_p, c_void_p, c_int32, c_int32, c_int32, c_int32, c_void_p, c_void_p, c_void_p, c_void_p,
                                 c_void_p]),
    "b200dec_dispatch": (c_int32, [c_void_p, c_int32, c_void_p, c_void_p, c_void_p, c_void_p, c_int32, c_int32, c_int32, c_int32, c_int32,
                                   c_void_p, c_void_p, c_void_p, c_void_p, c_int32, c_void_p]),
    "b200dec_grouped_linear": (c_int32, [c_void_p, c_void_p, c_int32, c_void_p, c_int32, c_int32, c_int32, c_int32, c_int32, c_int32,
                                         c_void_p, c_int32, c_float, c_float, c_void_p, c_int32, c_int32, c_void_p, c_void_p]),
}
SHARED_SIGNATURES = ("b200kv_version", "b200kv_error_string", "b200kv_set_chained_launch", "b200kv_get_chained_launch",
                     "b200kv_sample_workspace_bytes", "b200kv_sample")

_lib = None
_decoder_lib = None


class B200KVError(RuntimeError):
    pass


_path_override = None


def use_library(path: str) -> None:
    """Load this build of the library instead of the default one (the instrumented build of bench.py --phases).
    Must be called before the first op."""
    global _path_override
    if _lib is not None:
        raise B200KVError("a library is already loaded")
    _path_override = path


def load(build_if_needed: bool = True) -> C.CDLL:
    """Load (building first if sources are newer) the CUDA library.  Raises if impossible."""
    global _lib
    if _lib is not None:
        return _lib
    path = _build.LIB
    if build_if_needed and _build.needs_build():
        path = _build.build()
    if _path_override is not None:
        path = _path_override
    elif os.environ.get("B200KV_LIBRARY"):  # another build of the same sources (an experiment with other tile constants)
        path = os.environ["B200KV_LIBRARY"]
    if not os.path.exists(path):
        raise B200KVError(f"{path} is missing: the CUDA extension is required, there is no fallback path")
    lib = C.CDLL(path)
    for name, (res, args) in SIGNATURES.items():
        fn = getattr(lib, name, None)
        if fn is None:
            continue  # entry points are added unit by unit; exported_symbols() reports what exists
        fn.restype, fn.argtypes = res, args
    _lib = lib
    return lib


def load_decoder() -> C.CDLL:
    """Load (building first if sources are newer) libb200dec.so.  Raises if impossible."""
    global _decoder_lib
    if _decoder_lib is not None:
        return _decoder_lib
    lib = C.CDLL(_build.build_library(_build.DECODER_LIB))
    for name in SHARED_SIGNATURES:
        getattr(lib, name).restype, getattr(lib, name).argtypes = SIGNATURES[name]
    for name, (res, args) in DECODER_SIGNATURES.items():
        getattr(lib, name).restype, getattr(lib, name).argtypes = res, args
    _decoder_lib = lib
    return lib


def either() -> C.CDLL:
    """Whichever library is loaded already (the full one first), for the entry points both hold."""
    return _lib or _decoder_lib or load()


def check(rc: int, what: str) -> None:
    if rc != 0:
        msg = either().b200kv_error_string(rc)
        raise ValueError(f"{what}: {msg.decode() if msg else rc}")
