// Shared-memory barriers, tensor-map (TMA) loads and tensor-map encoding for the b200dec tensor-core kernels.
#pragma once
#include <cuda.h>  // CUtensorMap and the cuTensorMapEncodeTiled prototype only; the entry point is fetched at run time

#include "dec_common.cuh"

namespace b200kv {

constexpr uint32_t kDtSpin = 1u << 20;  // polls before a bounded wait gives up

__device__ __forceinline__ uint32_t dt_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void dt_mbar_init(uint32_t bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;\n" ::"r"(bar), "r"(count) : "memory");
}
// Bounded wait for the phase with the given parity; false when the limit ran out.
__device__ __forceinline__ bool dt_mbar_wait(uint32_t bar, uint32_t parity, uint32_t limit = kDtSpin) {
  for (uint32_t spin = 0; spin < limit; ++spin) {
    uint32_t done;
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}\n"
        : "=r"(done) : "r"(bar), "r"(parity) : "memory");
    if (done) return true;
  }
  return false;
}
__device__ __forceinline__ void dt_mbar_arrive(uint32_t bar) {
  asm volatile("{\n\t.reg .b64 st;\n\tmbarrier.arrive.shared::cta.b64 st, [%0];\n\t}\n" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void dt_expect_tx(uint32_t bar, uint32_t bytes) {
  asm volatile("{\n\t.reg .b64 st;\n\tmbarrier.arrive.expect_tx.shared::cta.b64 st, [%0], %1;\n\t}\n" ::"r"(bar), "r"(bytes) : "memory");
}
// Tile loads into this block alone.  The innermost coordinate is a multiple of 64 bf16 (128 bytes) everywhere, so every
// copy starts on a 16-byte boundary.
__device__ __forceinline__ void dt_tma_2d(uint32_t dst, const CUtensorMap* map, int c0, int c1, uint32_t bar) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];\n"
      ::"r"(dst), "l"(map), "r"(c0), "r"(c1), "r"(bar) : "memory");
}
__device__ __forceinline__ void dt_tma_3d(uint32_t dst, const CUtensorMap* map, int c0, int c1, int c2, uint32_t bar) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];\n"
      ::"r"(dst), "l"(map), "r"(c0), "r"(c1), "r"(c2), "r"(bar) : "memory");
}

typedef CUresult (*dt_encode_fn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                 const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                 CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
inline dt_encode_fn dt_encoder() {
  static dt_encode_fn fn = [] {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess)
      p = nullptr;
    return (dt_encode_fn)p;
  }();
  return fn;
}
// A bf16 tensor of `rank` dimensions (innermost first; strides in elements of dimensions 1..), read in boxes of 64
// channels x box rows with the 128-byte swizzle; what lies outside reads as zero.
inline bool dt_make_map(CUtensorMap* map, const void* base, int rank, const uint64_t* dims, const uint64_t* strides, const uint32_t* box) {
  dt_encode_fn enc = dt_encoder();
  if (!enc) return false;
  cuuint64_t d[5], st[4];
  cuuint32_t bx[5], es[5];
  for (int i = 0; i < rank; ++i) {
    if (dims[i] == 0) return false;
    d[i] = dims[i];
    bx[i] = box[i];
    es[i] = 1;
    if (i) st[i - 1] = strides[i - 1] * 2;
  }
  return enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void*>(base), d, st, bx, es, CU_TENSOR_MAP_INTERLEAVE_NONE,
             CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}
// Keys or values of a paged cache as [pages * heads][page_size][dim], read `rows` token rows at a time.
inline int dec_box_rows(int page_size) { return page_size % 64 == 0 ? 64 : (page_size % 32 == 0 ? 32 : 16); }
inline bool dt_cache_map(CUtensorMap* map, const void* base, int dim, int row, int page_size, long long page_heads, int rows) {
  const uint64_t dims[3] = {(uint64_t)dim, (uint64_t)page_size, (uint64_t)page_heads};
  const uint64_t strides[2] = {(uint64_t)row, (uint64_t)row * page_size};
  const uint32_t box[3] = {64, (uint32_t)rows, 1};
  return dt_make_map(map, base, 3, dims, strides, box);
}

}  // namespace b200kv
