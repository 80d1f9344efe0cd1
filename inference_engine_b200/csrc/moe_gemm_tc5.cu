// Grouped product of a mixture of experts on the 5th-generation tensor cores: y[row] = W_e x[row] for rows ordered by
// expert, cut into tiles of at most kN rows of one expert each (the list b200dec_dispatch writes).
//
// Roles as in skinny_linear_tc5.cu: 128 WEIGHT rows are the M dimension of tcgen05.mma (bf16 -> fp32), the tokens of a tile
// its N dimension, which follows the tile's row count in steps of 16, so a short tile costs only its own products.  The same
// kernel so serves prompts (kN = 256: M128 N256 K16, the full rate of the tensor core) and decode steps (kN = 64, where it
// streams the weights of the experts in use and the ring is twice as deep).
//   grid: one persistent CTA per SM; work items (tile, block of 128 weight rows), weight blocks fastest
//   warp 0, one lane   per 64 channels one TMA box of weights (128 rows, 16 KB) and the tile's rows of x in boxes of 64 or 16
//                      rows, into a ring of slots counted in bytes on `full`
//   warp 1, one lane   4 x tcgen05.mma per slot, commit on the slot's `empty`; after an item commit on `done[buffer]`
//   warps 2-5          epilogue from one of two accumulators in tensor memory (lane = weight row, column = token) while the
//                      other is being filled.  With the gated unit, gate and up rows of an output channel are neighbouring
//                      lanes and meet in one shuffle per two tokens; the token's score multiplies both (the experts'
//                      input is scaled, and the products are linear in it).
// Every wait is bounded; when one runs out its role stops, the CTA stores nothing more and sets B200KV_S_TIMEOUT.
#include "dec_tma.cuh"
#include "tmem_ldst.cuh"

namespace b200kv {

constexpr int kMgM = 128;       // weight rows per item
constexpr int kMgStep = 64;     // channels per slot
constexpr int kMgThreads = 192;
constexpr uint32_t kMgWBytes = kMgM * kMgStep * 2;  // 16 KB

template <int kN>
struct MgShape {
  static constexpr int kBox = kN == 256 ? 64 : 16;          // token rows per TMA box
  static constexpr int kStages = kN == 256 ? 4 : 8;
  static constexpr uint32_t kSlot = kMgWBytes + kN * kMgStep * 2;
  static constexpr uint32_t kCols = 2 * kN;                 // tensor-memory columns, two accumulators
  static constexpr size_t kSmem = kStages * kSlot + 1024 + 256;
};

__device__ __forceinline__ void mg_commit(uint32_t bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n" ::"r"(bar) : "memory");
}
// K-major operand in the 128-byte-swizzled layout a tensor-map copy writes: rows of 128 bytes, 8-row groups 1024 bytes apart
__device__ __forceinline__ uint64_t mg_desc(uint32_t saddr) {
  return (uint64_t)((saddr & 0x3FFFFu) >> 4) | ((uint64_t)(16u >> 4) << 16) | ((uint64_t)(1024u >> 4) << 32) | (1ull << 46) |
         (2ull << 61);
}
// kind::f16: fp32 accumulator, bf16 A and B (both K-major), M = 128, N = n
__device__ __forceinline__ uint32_t mg_idesc(uint32_t n) { return (1u << 4) | (1u << 7) | (1u << 10) | ((n >> 3) << 17) | ((128u >> 4) << 24); }
__device__ __forceinline__ void mg_mma(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}\n"
      ::"r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(acc) : "memory");
}

// Work item: a tile of one expert's rows and a block of its weight rows.  An entry of the list that does not fit (it would be
// the product of an inconsistent routing) is reported and passed over, alike by every role.
struct MgItem {
  int e, row0, rows, m0;
  bool ok;
};
template <int kN>
__device__ __forceinline__ MgItem mg_item(const int32_t* tiles, int it, int blocks, int experts, int total_rows) {
  const int t = it / blocks;
  MgItem x;
  x.m0 = (it - t * blocks) * kMgM;
  x.e = ld_fresh(tiles + 1 + 3 * t);
  x.row0 = ld_fresh(tiles + 2 + 3 * t);
  x.rows = ld_fresh(tiles + 3 + 3 * t);
  x.ok = x.e >= 0 && x.e < experts && x.rows >= 1 && x.rows <= kN && x.row0 >= 0 && x.row0 <= total_rows - x.rows;
  return x;
}

template <int kN, bool kAct>
__global__ void __launch_bounds__(kMgThreads, 1)
grouped_linear_tc5_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x, const int32_t* __restrict__ tiles,
                          int max_tiles, int experts, int total_rows, int out_rows, int steps, const float* __restrict__ score_sorted,
                          float limit, float slope, uint16_t* __restrict__ y, int32_t* status) {
  using S = MgShape<kN>;
  extern __shared__ uint8_t mg_raw[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t base = (dt_smem(mg_raw) + 1023u) & ~1023u;
  const uint32_t bars = base + S::kStages * S::kSlot;
  auto bar_full = [&](int s) { return bars + 8 * s; };
  auto bar_empty = [&](int s) { return bars + 8 * (S::kStages + s); };
  auto bar_done = [&](int b) { return bars + 16 * S::kStages + 8 * b; };        // accumulator b is complete
  auto bar_free = [&](int b) { return bars + 16 * S::kStages + 16 + 8 * b; };   // ... and read (4 epilogue warps)
  const uint32_t slot_word = bars + 16 * S::kStages + 32;
  if (tid == 0) {
    for (int s = 0; s < S::kStages; ++s) {
      dt_mbar_init(bar_full(s), 1);
      dt_mbar_init(bar_empty(s), 1);
    }
    for (int b = 0; b < 2; ++b) {
      dt_mbar_init(bar_done(b), 1);
      dt_mbar_init(bar_free(b), 4);
    }
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(slot_word), "r"(S::kCols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
  uint32_t tmem;
  asm volatile("ld.shared.u32 %0, [%1];\n" : "=r"(tmem) : "r"(slot_word) : "memory");
  pdl_wait();  // the tile list and the rows come from the kernels before this one
  const int blocks = (out_rows + kMgM - 1) / kMgM;
  const int items = min(max(ld_fresh(tiles), 0), max_tiles) * blocks;

  if (warp == 0) {
    if (lane == 0) {
      int i = 0;
      bool live = true;
      for (int it = blockIdx.x; it < items && live; it += gridDim.x) {
        const MgItem x = mg_item<kN>(tiles, it, blocks, experts, total_rows);
        if (!x.ok) {
          if (status) atomicOr(status, B200KV_S_BAD_POSITION);
          continue;
        }
        const int boxes = (x.rows + S::kBox - 1) / S::kBox;
        const uint32_t bytes = kMgWBytes + (uint32_t)boxes * S::kBox * 128;
        for (int k = 0; k < steps; ++k, ++i) {
          const int s = i % S::kStages;
          if (i >= S::kStages && !dt_mbar_wait(bar_empty(s), (i / S::kStages - 1) & 1)) { live = false; break; }
          const uint32_t dst = base + s * S::kSlot;
          dt_expect_tx(bar_full(s), bytes);
          dt_tma_2d(dst, &tm_w, k * kMgStep, x.e * out_rows + x.m0, bar_full(s));
          for (int b = 0; b < boxes; ++b) dt_tma_2d(dst + kMgWBytes + b * S::kBox * 128, &tm_x, k * kMgStep, x.row0 + b * S::kBox, bar_full(s));
        }
      }
      pdl_trigger();  // nothing left to fetch: the next kernel may be brought up
      if (!live) {    // the copies in flight land before the CTA may end
        if (status) atomicOr(status, B200KV_S_TIMEOUT);
        for (int k = i > S::kStages ? i - S::kStages : 0; k < i; ++k) dt_mbar_wait(bar_full(k % S::kStages), (k / S::kStages) & 1);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      int i = 0, n = 0;
      bool live = true;
      for (int it = blockIdx.x; it < items && live; it += gridDim.x) {
        const MgItem x = mg_item<kN>(tiles, it, blocks, experts, total_rows);
        if (!x.ok) continue;
        const int buf = n & 1;
        const uint32_t idesc = mg_idesc((uint32_t)((x.rows + 15) & ~15));
        if (n >= 2 && !dt_mbar_wait(bar_free(buf), (n / 2 - 1) & 1)) break;
        asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
        for (int k = 0; k < steps; ++k, ++i) {
          const int s = i % S::kStages;
          if (!dt_mbar_wait(bar_full(s), (i / S::kStages) & 1)) { live = false; break; }
          asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
          const uint64_t da = mg_desc(base + s * S::kSlot), db = mg_desc(base + s * S::kSlot + kMgWBytes);
#pragma unroll
          for (int j = 0; j < kMgStep / 16; ++j)
            mg_mma(tmem + buf * kN, da + (uint64_t)((j * 32) >> 4), db + (uint64_t)((j * 32) >> 4), idesc, (k | j) != 0);
          mg_commit(bar_empty(s));
        }
        if (live) mg_commit(bar_done(buf));
        ++n;
      }
    }
  } else {
    int n = 0;
    const int wl = warp & 3;  // tensor-memory lanes 32 wl ..
    for (int it = blockIdx.x; it < items; it += gridDim.x) {
      const MgItem x = mg_item<kN>(tiles, it, blocks, experts, total_rows);
      if (!x.ok) continue;
      const int buf = n & 1, row0 = x.row0, rows = x.rows;
      const int o = x.m0 + 32 * wl + lane;  // this lane's weight row
      const bool ok = dt_mbar_wait(bar_done(buf), (n / 2) & 1);
      if (!__all_sync(0xffffffffu, ok)) {
        if (lane == 0 && status) atomicOr(status, B200KV_S_TIMEOUT);
        break;
      }
      asm volatile("tcgen05.fence::after_thread_sync;\n" ::: "memory");
      for (int c0 = 0; c0 < rows; c0 += 32) {
        uint32_t u[32];
        t5_ld32(tmem + buf * kN + c0 + ((uint32_t)(32 * wl) << 16), u);
        if (kAct) {
          const float sl = c0 + lane < rows ? ld_fresh(score_sorted + row0 + c0 + lane) : 0.f;
          const bool odd = lane & 1;
          uint16_t* dst = y + (long long)(row0 + c0 + odd) * (out_rows / 2) + o / 2;
#pragma unroll
          for (int c = 0; c < 32; c += 2) {
            const float a = __uint_as_float(u[c]) * __shfl_sync(0xffffffffu, sl, c);
            const float b = __uint_as_float(u[c + 1]) * __shfl_sync(0xffffffffu, sl, c + 1);
            const float got = __shfl_xor_sync(0xffffffffu, odd ? a : b, 1);
            const float g = fminf(odd ? got : a, limit), up = fminf(fmaxf(odd ? b : got, -limit), limit);
            const float v = __fdividef(g, 1.0f + __expf(-slope * g)) * (up + 1.0f);
            if (c0 + c + odd < rows && o < out_rows) *dst = (uint16_t)float_to_bf16_bits(v);
            dst += out_rows;  // two tokens further: 2 * (out_rows / 2)
          }
        } else {
          uint16_t* dst = y + (long long)(row0 + c0) * out_rows + o;
#pragma unroll
          for (int c = 0; c < 32; ++c) {
            if (c0 + c < rows && o < out_rows) *dst = (uint16_t)float_to_bf16_bits(__uint_as_float(u[c]));
            dst += out_rows;
          }
        }
      }
      asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
      __syncwarp();
      if (lane == 0) dt_mbar_arrive(bar_free(buf));
      ++n;
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;\n" ::: "memory");
  __syncthreads();
  if (warp == 0) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(S::kCols) : "memory");
}

template <int kN, bool kAct>
static int mg_launch(const CUtensorMap& tm_w, const CUtensorMap& tm_x, const int32_t* tiles, int grid, int max_tiles, int experts, int total_rows, int out_rows, int steps,
                     const float* score_sorted, float limit, float slope, void* y, int32_t* status, cudaStream_t stream) {
  if (cudaFuncSetAttribute(grouped_linear_tc5_kernel<kN, kAct>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MgShape<kN>::kSmem) !=
      cudaSuccess)
    return B200KV_E_LAUNCH;
  return launch_result(launch_chained(grouped_linear_tc5_kernel<kN, kAct>, dim3(grid), dim3(kMgThreads), MgShape<kN>::kSmem, stream, tm_w, tm_x,
                                      tiles, max_tiles, experts, total_rows, out_rows, steps, score_sorted, limit, slope, (uint16_t*)y, status));
}

int launch_grouped_linear_tc5(const void* x, const void* w, const int32_t* tiles, int max_tiles, int tile_rows, int total_rows, int experts,
                              int out_rows, int width, const float* score_sorted, int act, float limit, float slope, void* y, int sms,
                              int32_t* status, cudaStream_t stream) {
  if (tile_rows > 256) return B200KV_E_SHAPE;
  if ((long long)experts * out_rows > 0x7FFFFFFFll) return B200KV_E_RANGE;
  const int box = tile_rows > 64 ? MgShape<256>::kBox : MgShape<64>::kBox;
  CUtensorMap tm_w, tm_x;
  const uint64_t wd[2] = {(uint64_t)width, (uint64_t)experts * out_rows}, xd[2] = {(uint64_t)width, (uint64_t)total_rows};
  const uint64_t st[1] = {(uint64_t)width};
  const uint32_t wb[2] = {kMgStep, kMgM}, xb[2] = {kMgStep, (uint32_t)box};
  if (!dt_make_map(&tm_w, w, 2, wd, st, wb) || !dt_make_map(&tm_x, x, 2, xd, st, xb)) return B200KV_E_LAUNCH;
  const long long items = (long long)max_tiles * ((out_rows + kMgM - 1) / kMgM);
  const int grid = (int)(items < sms ? items : sms), steps = (width + kMgStep - 1) / kMgStep;
  if (tile_rows > 64)
    return act ? mg_launch<256, true>(tm_w, tm_x, tiles, grid, max_tiles, experts, total_rows, out_rows, steps, score_sorted, limit, slope, y, status, stream)
               : mg_launch<256, false>(tm_w, tm_x, tiles, grid, max_tiles, experts, total_rows, out_rows, steps, score_sorted, limit, slope, y, status, stream);
  return act ? mg_launch<64, true>(tm_w, tm_x, tiles, grid, max_tiles, experts, total_rows, out_rows, steps, score_sorted, limit, slope, y, status, stream)
             : mg_launch<64, false>(tm_w, tm_x, tiles, grid, max_tiles, experts, total_rows, out_rows, steps, score_sorted, limit, slope, y, status, stream);
}

}  // namespace b200kv
