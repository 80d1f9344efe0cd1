// Host side of the tcgen05 prefill attention over [dequantized prefix | own chunk] (prefill_attn_tc5.cuh).
#include "prefill_attn_tc5.cuh"

namespace b200kv {

// cuTensorMapEncodeTiled, fetched from the driver through the runtime (the library links no libcuda).
typedef CUresult (*t5_encode_fn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                 const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                 CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
static t5_encode_fn t5_encoder() {
  static t5_encode_fn fn = [] {
    void* p = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess || q != cudaDriverEntryPointSuccess)
      p = nullptr;
    return (t5_encode_fn)p;
  }();
  return fn;
}
// A bf16 tensor [d2][d1][128 channels] with element strides (s2, s1, 1), read in boxes of 64 channels x b1 x b2
// with the 128-byte swizzle; out-of-range rows read as zero.
static bool t5_make_map(CUtensorMap* map, const void* base, uint64_t d1, uint64_t d2, long long s1, long long s2, uint32_t b1,
                        uint32_t b2) {
  t5_encode_fn enc = t5_encoder();
  if (!enc || d1 == 0 || d2 == 0 || s1 <= 0 || s2 <= 0) return false;
  const cuuint64_t dims[3] = {(cuuint64_t)kD, d1, d2};
  const cuuint64_t strides[2] = {(cuuint64_t)s1 * 2, (cuuint64_t)s2 * 2};
  const cuuint32_t box[3] = {64, b1, b2}, estr[3] = {1, 1, 1};
  return enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
             CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
             CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// prefix_rows: rows each kv head of k_prefix / v_prefix holds (0 = not known: prefix tiles are then copied with
// cp.async only).
int launch_prefill_attn_tc5(const uint16_t* q, long long q_sn, long long q_sh, const uint16_t* k, long long k_sn,
                            long long k_sh, const uint16_t* v, long long v_sn, long long v_sh, const int32_t* seq_ids,
                            const int32_t* cu_seqlens, const int32_t* tile_start, int num_tiles, int block_m,
                            const uint16_t* k_prefix, const uint16_t* v_prefix, long long p_sh, long long p_sn,
                            int prefix_rows, const int32_t* cu_cached, uint16_t* out, long long o_sn, long long o_sh, int N,
                            int Hq, int Hkv, float scale_log2, int32_t* status, int idle_issuers, cudaStream_t stream) {
  // the opt-in is a per-device attribute of the function: set it on every call (it is cheap)
  if (cudaFuncSetAttribute(prefill_attn_tc5_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kT5Smem) !=
      cudaSuccess)
    return B200KV_E_LAUNCH;
  CUtensorMap tm_k, tm_v, tm_kp, tm_vp;
  // own chunk [N][Hkv][128]: box = 64 rows of one head
  if (!t5_make_map(&tm_k, k, Hkv, N, k_sh, k_sn, 1, kT5Keys) || !t5_make_map(&tm_v, v, Hkv, N, v_sh, v_sn, 1, kT5Keys))
    return B200KV_E_LAUNCH;
  // prefix [Hkv][rows][128]: box = 64 rows of one head; without a row count the maps are placeholders
  int prefix_tma = prefix_rows > 0 && t5_make_map(&tm_kp, k_prefix, prefix_rows, Hkv, p_sn, p_sh, kT5Keys, 1) &&
                   t5_make_map(&tm_vp, v_prefix, prefix_rows, Hkv, p_sn, p_sh, kT5Keys, 1);
  if (!prefix_tma) { tm_kp = tm_k; tm_vp = tm_v; }
  const int subs = (block_m + kT5Tile - 1) / kT5Tile;
  const cudaError_t le = launch_chained(prefill_attn_tc5_kernel<false>, dim3(Hq, num_tiles * subs), dim3(kT5Threads), kT5Smem, stream,
                                        q, q_sn, q_sh, k, k_sn, k_sh, v, v_sn, v_sh, seq_ids, cu_seqlens, tile_start, block_m, subs,
                                        k_prefix, v_prefix, p_sh, p_sn, cu_cached, out, o_sn, o_sh, N, Hq / Hkv, scale_log2, status,
                                        tm_k, tm_v, tm_kp, tm_vp, prefix_tma, idle_issuers, T5Paged{});
  return le == cudaSuccess && cudaGetLastError() == cudaSuccess ? B200KV_OK : B200KV_E_LAUNCH;
}

}  // namespace b200kv
