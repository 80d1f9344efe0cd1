"""Builds the C-ABI CUDA libraries in-tree with nvcc for sm_100a.

    python -m inference_engine_b200.build [--force]

libb200kv.so holds the int8-cache attention path and the ops around it (include/b200kv.h), libb200dec.so the decoder ops
in the model's own precision (include/b200dec.h) with the sampler and the status words, so that serving a model of that
kind needs the second library only.  Units are compiled side by side, and only when they changed.

The write-path translation unit is compiled with -fmad=false: its results must be bit-identical
to separately rounded IEEE fp32 arithmetic.  There is no other backend and no fallback: if the
library cannot be built or loaded the package raises.
"""
from __future__ import annotations

import os
import shutil
import subprocess
import sys
from concurrent.futures import ThreadPoolExecutor

PKG = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(PKG)
CSRC = os.path.join(PKG, "csrc")
INCLUDE = os.path.join(ROOT, "include")
LIB = os.path.join(PKG, "libb200kv.so")
OBJ_DIR = os.path.join(PKG, "build")

ARCH = ["-gencode", "arch=compute_100a,code=sm_100a"]
COMMON = ["-O3", "-lineinfo", "-std=c++17", "-Xcompiler", "-fPIC", "-I", INCLUDE, "-I", CSRC]
UNITS = {  # unit -> extra flags
    "abi.cu": [],
    "write_kernels.cu": ["-fmad=false"],
    "decode_attn.cu": [],
    "prefill_attn.cu": [],
    "prefill_attn_tc5.cu": [],
    "block_ops.cu": [],
    "sampler.cu": ["-fmad=false"],
    "skinny_linear_tc5.cu": [],
    "row_ops.cu": [],
    "paged_rows.cu": [],
    "paged_decode.cu": [],
    "paged_prefill_tc5.cu": [],
    "moe.cu": [],
    "moe_gemm_tc5.cu": [],
    "recurrence.cu": [],
    "recurrence_decode.cu": [],
    "recurrence_block.cu": [],
    "ssd_scan.cu": [],
}
DECODER_LIB = os.path.join(PKG, "libb200dec.so")
LIBRARIES = {
    LIB: ["abi.cu", "write_kernels.cu", "decode_attn.cu", "prefill_attn.cu", "prefill_attn_tc5.cu", "block_ops.cu", "sampler.cu",
          "skinny_linear_tc5.cu"],
    DECODER_LIB: ["abi.cu", "sampler.cu", "paged_prefill_tc5.cu", "row_ops.cu", "paged_rows.cu", "paged_decode.cu", "moe.cu", "moe_gemm_tc5.cu",
                  "recurrence.cu", "recurrence_decode.cu", "recurrence_block.cu", "ssd_scan.cu"],
}
# The same library with per-warp timestamps compiled into the decode-attention kernel (bench.py --phases);
# never loaded by the product path.
STAMPS_LIB = os.path.join(PKG, "libb200kv_stamps.so")


def _nvcc() -> str:
    for cand in (os.environ.get("NVCC"), shutil.which("nvcc"), "/usr/local/cuda/bin/nvcc"):
        if cand and os.path.exists(cand):
            return cand
    raise RuntimeError("nvcc not found: libb200kv.so cannot be built")


def headers() -> list[str]:
    return sorted([os.path.join(d, f) for d in (CSRC, INCLUDE) for f in os.listdir(d) if f.endswith((".cuh", ".h"))])


def _newer(deps: list[str], target: str) -> bool:
    if not os.path.exists(target):
        return True
    t = os.path.getmtime(target)
    return any(os.path.getmtime(d) > t for d in deps)


def needs_build(lib: str = LIB) -> bool:
    return _newer([os.path.join(CSRC, u) for u in LIBRARIES[lib]] + headers(), lib)


def _compile(unit: str, force: bool, verbose: bool) -> str:
    src, obj = os.path.join(CSRC, unit), os.path.join(OBJ_DIR, unit.replace(".cu", ".o"))
    if force or _newer([src] + headers(), obj):
        tmp = f"{obj}.{os.getpid()}"
        cmd = [_nvcc(), *ARCH, *COMMON, *UNITS[unit], "-c", src, "-o", tmp]
        if verbose:
            cmd.insert(1, "-Xptxas=-v")
        subprocess.run(cmd, check=True, stdout=sys.stderr if not verbose else None)
        os.replace(tmp, obj)
    return obj


def build_library(lib: str, force: bool = False, verbose: bool = False) -> str:
    """One library, with the units it needs and no others."""
    if not force and not needs_build(lib):
        return lib
    os.makedirs(OBJ_DIR, exist_ok=True)
    with ThreadPoolExecutor(max_workers=max(1, min(8, os.cpu_count() or 1))) as pool:
        objs = list(pool.map(lambda u: _compile(u, force, verbose), LIBRARIES[lib]))
    tmp = f"{lib}.{os.getpid()}"
    subprocess.run([_nvcc(), *ARCH, "-shared", "-cudart", "static", "-o", tmp, *objs], check=True)
    os.replace(tmp, lib)
    return lib


def build(force: bool = False, verbose: bool = False) -> str:
    """Every library (and the instrumented one of bench.py --phases).  Returns the path of libb200kv.so."""
    stale = force or needs_build(LIB) or not os.path.exists(STAMPS_LIB)
    build_library(DECODER_LIB, force, verbose)
    build_library(LIB, force, verbose)
    if stale:
        build_stamps(_nvcc(), [os.path.join(OBJ_DIR, u.replace(".cu", ".o")) for u in LIBRARIES[LIB]])
    return LIB


def build_stamps(nvcc: str, objs: list[str]) -> str:
    """libb200kv_stamps.so = the library with decode_attn.cu recompiled under -DB200KV_STAMPS."""
    obj = os.path.join(OBJ_DIR, "decode_attn_stamps.o")
    subprocess.run([nvcc, *ARCH, *COMMON, "-DB200KV_STAMPS", "-c", os.path.join(CSRC, "decode_attn.cu"), "-o", obj], check=True)
    rest = [o for o in objs if os.path.basename(o) != "decode_attn.o"]
    tmp = STAMPS_LIB + ".tmp"
    subprocess.run([nvcc, *ARCH, "-shared", "-cudart", "static", "-o", tmp, *rest, obj], check=True)
    os.replace(tmp, STAMPS_LIB)
    return STAMPS_LIB


if __name__ == "__main__":
    print(build(force="--force" in sys.argv, verbose="-v" in sys.argv))
