// Host side of the tcgen05 prefill attention over the paged bf16 cache (prefill_attn_tc5.cuh).
#include "dec_tma.cuh"
#include "prefill_attn_tc5.cuh"

using namespace b200kv;

extern "C" int b200dec_prefill_attn_opt(const void* q, const b200dec_cache* cache, const b200kv_table* table, const int32_t* seq_ids,
                                        const int32_t* cu_seqlens, const int32_t* cached_lens, const int32_t* tile_start,
                                        int32_t num_tiles, int32_t block_m, int32_t num_rows, int32_t heads, float scale,
                                        const b200dec_attn_options* options, void* out, int32_t* status, void* stream) {
  if (num_rows == 0 || num_tiles == 0) return B200KV_OK;
  if (!q || !seq_ids || !cu_seqlens || !cached_lens || !tile_start || !out) return B200KV_E_NULL;
  const int rc = check_dec_cache(cache, table);
  if (rc != B200KV_OK) return rc;
  if (cache->elem != 2 || cache->k_dim > kD || cache->v_dim > kD || cache->page_size % 16 || heads < 1 || heads % cache->kv_heads ||
      num_rows < 0 || num_tiles < 0 || block_m < 1)
    return B200KV_E_SHAPE;
  const int subs = (block_m + kT5Tile - 1) / kT5Tile;
  if ((long long)num_tiles * subs > 65535 || (long long)cache->num_pages * cache->kv_heads > 0x7FFFFFFFll) return B200KV_E_RANGE;
  if (!aligned(q, 16) || !aligned(out, 16)) return B200KV_E_ALIGN;
  T5Paged pg;
  const int bad = dec_attn_opt(options, heads, cache->v_dim, &pg.opt);
  if (bad != B200KV_OK) return bad;
  pg.c = dec_view(cache, table);
  pg.cached_lens = cached_lens;
  pg.box_rows = dec_box_rows(pg.c.P);
  CUtensorMap tm_k, tm_v;
  const long long ph = (long long)pg.c.num_pages * pg.c.heads;
  if (!dt_cache_map(&tm_k, pg.c.k, pg.c.k_dim, pg.c.k_row, pg.c.P, ph, pg.box_rows) ||
      !dt_cache_map(&tm_v, pg.c.v, pg.c.v_dim, pg.c.v_row, pg.c.P, ph, pg.box_rows))
    return B200KV_E_LAUNCH;
  const bool two = pg.c.k_dim > 64;
  auto kernel = options ? (two ? prefill_attn_tc5_kernel<true, 2, true> : prefill_attn_tc5_kernel<true, 1, true>)
                        : (two ? prefill_attn_tc5_kernel<true, 2> : prefill_attn_tc5_kernel<true, 1>);
  // the opt-in is a per-device attribute of the function: set it on every call (it is cheap)
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kT5Smem) != cudaSuccess) return B200KV_E_LAUNCH;
  const uint16_t* none = nullptr;
  const int32_t* no_lens = nullptr;
  return launch_result(launch_chained(
      kernel, dim3(heads, num_tiles * subs), dim3(kT5Threads), kT5Smem, (cudaStream_t)stream, (const uint16_t*)q,
      (long long)heads * pg.c.k_row, (long long)pg.c.k_row, none, 0LL, 0LL, none, 0LL, 0LL, seq_ids, cu_seqlens, tile_start, block_m, subs, none,
      none, 0LL, 0LL, no_lens, (uint16_t*)out, pg.opt.out_stride, (long long)pg.c.v_dim, num_rows, heads / pg.c.heads,
      scale * 1.4426950408889634f, status, tm_k, tm_v, tm_k, tm_v, 0, 0, pg));
}

extern "C" int b200dec_prefill_attn(const void* q, const b200dec_cache* cache, const b200kv_table* table, const int32_t* seq_ids,
                                    const int32_t* cu_seqlens, const int32_t* cached_lens, const int32_t* tile_start, int32_t num_tiles,
                                    int32_t block_m, int32_t num_rows, int32_t heads, float scale, void* out, int32_t* status, void* stream) {
  return b200dec_prefill_attn_opt(q, cache, table, seq_ids, cu_seqlens, cached_lens, tile_start, num_tiles, block_m, num_rows, heads, scale,
                                  nullptr, out, status, stream);
}
