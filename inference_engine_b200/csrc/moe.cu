// Mixture of experts: the router (32-bit scores, top choices, a place for every choice), the layout of tokens by
// expert, and the grouped product on the CUDA cores (any sizes, fp32 or bf16; the tensor-core one is
// moe_gemm_tc5.cu).
#include "dec_common.cuh"

namespace b200kv {

// ------------------------------------------------------------------ router
// One block per kR rows, which it keeps in shared memory.  A warp takes four experts at a time and, when there are fewer
// groups of four than warps, a slice of the channels of them; its lanes run over the channels, so a weight is read once
// per kR rows and a channel of x once per four experts.
constexpr int kRtWarps = 8;
constexpr int kRtExperts = 4;
constexpr int kRtMaxExperts = 1024;

template <int kR>
__global__ void __launch_bounds__(kRtWarps * 32, 4)
router_kernel(const float* __restrict__ x, const uint16_t* __restrict__ w, int N, int width, int E, int top, int slices,
              int32_t* __restrict__ ids, float* __restrict__ scores, int32_t* __restrict__ ranks, int32_t* __restrict__ counts) {
  extern __shared__ __align__(16) float rt_smem[];
  const int pitch = (width + 3) & ~3;
  float* xs = rt_smem;                // [kR][pitch]
  float* sc = xs + kR * pitch;        // [kR][E]
  float* part = sc + kR * E;          // [slices][kR][E], only with slices > 1
  pdl_enter();
  pdl_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r0 = blockIdx.x * kR, nr = min(kR, N - r0);
  for (int r = 0; r < kR; ++r) {
    const float* src = x + (long long)(r0 + r) * width;
    if (width % 4 == 0) {
      for (int c = tid * 4; c < width; c += kRtWarps * 128) {
        float f[4] = {0.f, 0.f, 0.f, 0.f};
        if (r < nr) ld_fresh4(src + c, f);
        st_elem4(xs + r * pitch + c, f);
      }
    } else {
      for (int c = tid; c < width; c += kRtWarps * 32) xs[r * pitch + c] = r < nr ? ld_fresh(src + c) : 0.f;
    }
  }
  __syncthreads();
  const int groups = (E + kRtExperts - 1) / kRtExperts;
  for (int item = warp; item < groups * slices; item += kRtWarps) {
    const int e0 = item / slices * kRtExperts, slice = item % slices;
    float acc[kRtExperts][kR];
#pragma unroll
    for (int i = 0; i < kRtExperts; ++i)
#pragma unroll
      for (int r = 0; r < kR; ++r) acc[i][r] = 0.f;
    const uint16_t* wp[kRtExperts];
#pragma unroll
    for (int i = 0; i < kRtExperts; ++i) wp[i] = w + (long long)min(e0 + i, E - 1) * width;
    if (width % 4 == 0) {
      const int per = (width / 4 + slices - 1) / slices * 4, hi = min(width, (slice + 1) * per);
#pragma unroll 2
      for (int c = slice * per + 4 * lane; c < hi; c += 128) {
        float wv[kRtExperts][4];
#pragma unroll
        for (int i = 0; i < kRtExperts; ++i) ld_elem4(wp[i] + c, wv[i]);
#pragma unroll
        for (int r = 0; r < kR; ++r) {
          float xv[4];
          ld_elem4(xs + r * pitch + c, xv);
#pragma unroll
          for (int i = 0; i < kRtExperts; ++i)
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[i][r] = fmaf(wv[i][k], xv[k], acc[i][r]);
        }
      }
    } else {
      for (int c = slice * 32 + lane; c < width; c += 32 * slices)
#pragma unroll
        for (int i = 0; i < kRtExperts; ++i)
#pragma unroll
          for (int r = 0; r < kR; ++r) acc[i][r] = fmaf(ld_elem(wp[i] + c), xs[r * pitch + c], acc[i][r]);
    }
    float* dst = slices > 1 ? part + slice * kR * E : sc;
#pragma unroll
    for (int i = 0; i < kRtExperts; ++i)
#pragma unroll
      for (int r = 0; r < kR; ++r) {
        const float z = warp_sum(acc[i][r]);
        if (lane == 0 && e0 + i < E) dst[r * E + e0 + i] = z;
      }
  }
  __syncthreads();
  for (int i = tid; i < kR * E; i += kRtWarps * 32) {
    float z = 0.f;
    if (slices > 1)
      for (int k = 0; k < slices; ++k) z += part[k * kR * E + i];
    else
      z = sc[i];
    // a score that is not a number (an idle row's left-overs) counts as the smallest one
    sc[i] = z == z ? 1.0f / (1.0f + expf(-z)) : 0.f;
  }
  __syncthreads();
  for (int r = warp; r < nr; r += kRtWarps) {
    float* s = sc + r * E;
    for (int j = 0; j < top; ++j) {
      float best = -1.f;
      int at = E;
      for (int e = lane; e < E; e += 32)
        if (s[e] > best) { best = s[e]; at = e; }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, at, o);
        if (ov > best || (ov == best && oi < at)) { best = ov; at = oi; }
      }
      if (lane == 0) {
        s[at] = -2.f;
        const long long o = (long long)(r0 + r) * top + j;
        ids[o] = at;
        scores[o] = best;
        ranks[o] = atomicAdd(counts + at, 1);
      }
      __syncwarp();
    }
  }
}

// ------------------------------------------------------------------ dispatch
constexpr int kDpThreads = 128;

// Exclusive prefix of v over the block (kDpThreads values); total in *sum.
__device__ __forceinline__ int dp_scan(int v, int* shared, int* sum) {
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  int incl = v;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int y = __shfl_up_sync(0xffffffffu, incl, o);
    if (lane >= o) incl += y;
  }
  __syncthreads();
  if (lane == 31) shared[warp] = incl;
  __syncthreads();
  int before = 0, tot = 0;
#pragma unroll
  for (int i = 0; i < kDpThreads / 32; ++i) {
    if (i < warp) before += shared[i];
    tot += shared[i];
  }
  *sum = tot;
  return before + incl - v;
}

// Blocks stride over the rows; every block scans the counts (experts <= 1024) for the experts' first places, block 0
// also writes the tile list.
template <typename T>
__global__ void __launch_bounds__(kDpThreads)
dispatch_kernel(const T* __restrict__ xb, const int32_t* __restrict__ ids, const float* __restrict__ scores,
                const int32_t* __restrict__ ranks, const int32_t* __restrict__ counts, int N, int width, int E, int top, int tile_rows,
                T* __restrict__ x_sorted, float* __restrict__ score_sorted, int32_t* __restrict__ slots, int32_t* __restrict__ tiles,
                int max_tiles) {
  __shared__ int first[kRtMaxExperts];
  __shared__ int red[kDpThreads / 32];
  pdl_enter();
  pdl_wait();
  const int tid = threadIdx.x;
  int base = 0, tbase = 0;
  for (int e0 = 0; e0 < E; e0 += kDpThreads) {
    const int e = e0 + tid, n = e < E ? ld_fresh(counts + e) : 0;
    int sum;
    const int f = base + dp_scan(n, red, &sum);
    base += sum;
    if (e < E) first[e] = f;
    if (blockIdx.x == 0) {
      // an expert's run is cut evenly: a short last tile would cost almost as much as a full one
      int nt = (n + tile_rows - 1) / tile_rows;
      const int each = nt ? min(tile_rows, ((n + nt - 1) / nt + 15) / 16 * 16) : 1;
      nt = (n + each - 1) / each;
      int t = tbase + dp_scan(nt, red, &sum);
      tbase += sum;
      for (int i = 0; i < nt && t < max_tiles; ++i, ++t) {
        tiles[1 + 3 * t] = e;
        tiles[2 + 3 * t] = f + i * each;
        tiles[3 + 3 * t] = min(each, n - i * each);
      }
    }
  }
  if (blockIdx.x == 0 && tid == 0) tiles[0] = min(tbase, max_tiles);
  __syncthreads();
  constexpr int kVec = 16 / sizeof(T);
  for (long long r = blockIdx.x; r < N; r += gridDim.x) {
    const T* src = xb + r * width;
    for (int j = 0; j < top; ++j) {
      const long long o = r * top + j;
      const int place = first[ld_fresh(ids + o)] + ld_fresh(ranks + o);
      T* dst = x_sorted + (long long)place * width;
      if (width % kVec == 0) {
        for (int c = tid * kVec; c < width; c += kDpThreads * kVec) *reinterpret_cast<uint4*>(dst + c) = *reinterpret_cast<const uint4*>(src + c);
      } else {
        for (int c = tid; c < width; c += kDpThreads) dst[c] = src[c];
      }
      if (tid == 0) {
        slots[o] = place;
        score_sorted[place] = ld_fresh(scores + o);
      }
    }
  }
}

// ------------------------------------------------------------------ grouped product on the CUDA cores
// 32 rows x 64 outputs per block, 16 channels per step; a thread computes 8 rows of one output.
constexpr int kGsRows = 32, kGsCols = 64, kGsStep = 16, kGsThreads = 256;

// y = g * sigmoid(slope * g) * (u + 1) with both inputs limited
__device__ __forceinline__ float gated_unit(float g, float u, float limit, float slope) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.0f + expf(-slope * g)) * (u + 1.0f);
}

template <typename T>
__global__ void __launch_bounds__(kGsThreads)
grouped_linear_simt_kernel(const T* __restrict__ x, const T* __restrict__ w, const int32_t* __restrict__ tiles, int out_rows, int width,
                           const float* __restrict__ score_sorted, int act, float limit, float slope, T* __restrict__ y) {
  __shared__ float xs[kGsStep][kGsRows + 1];
  __shared__ float ws[kGsStep][kGsCols + 1];
  pdl_enter();
  pdl_wait();
  const int num = ld_fresh(tiles), tid = threadIdx.x, col = tid & 63, rg = tid >> 6;
  const int o = blockIdx.x * kGsCols + col;
  for (int t = blockIdx.y; t < num; t += gridDim.y) {
    const int e = ld_fresh(tiles + 1 + 3 * t), row0 = ld_fresh(tiles + 2 + 3 * t), nrows = ld_fresh(tiles + 3 + 3 * t);
    for (int sub = 0; sub < nrows; sub += kGsRows) {
      const int n = min(kGsRows, nrows - sub);
      float acc[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[i] = 0.f;
      for (int c0 = 0; c0 < width; c0 += kGsStep) {
        __syncthreads();
        for (int i = tid; i < kGsRows * kGsStep; i += kGsThreads) {
          const int rr = i / kGsStep, c = i % kGsStep;
          xs[c][rr] = rr < n && c0 + c < width ? ld_elem(x + (long long)(row0 + sub + rr) * width + c0 + c) : 0.f;
        }
        for (int i = tid; i < kGsCols * kGsStep; i += kGsThreads) {
          const int cc = i / kGsStep, c = i % kGsStep, oo = blockIdx.x * kGsCols + cc;
          ws[c][cc] = oo < out_rows && c0 + c < width ? ld_elem(w + ((long long)e * out_rows + oo) * width + c0 + c) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < kGsStep; ++c) {
          const float wv = ws[c][col];
#pragma unroll
          for (int i = 0; i < 8; ++i) acc[i] = fmaf(wv, xs[c][rg * 8 + i], acc[i]);
        }
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int rr = rg * 8 + i;
        const long long row = row0 + sub + rr;
        if (act) {  // neighbouring lanes hold gate (even output) and up (odd output)
          const float s = rr < n ? ld_fresh(score_sorted + row) : 0.f;
          const float mine = acc[i] * s, other = __shfl_xor_sync(0xffffffffu, mine, 1);
          if (rr < n && o < out_rows && (o & 1) == 0) st_elem(y + row * (out_rows / 2) + o / 2, gated_unit(mine, other, limit, slope));
        } else if (rr < n && o < out_rows) {
          st_elem(y + row * out_rows + o, acc[i]);
        }
      }
    }
  }
}

int launch_grouped_linear_tc5(const void* x, const void* w, const int32_t* tiles, int max_tiles, int tile_rows, int total_rows, int experts,
                              int out_rows, int width, const float* score_sorted, int act, float limit, float slope, void* y, int sms,
                              int32_t* status, cudaStream_t stream);

}  // namespace b200kv

using namespace b200kv;

extern "C" int b200dec_router(const float* x, const void* router_w, int32_t num_rows, int32_t width, int32_t experts, int32_t top,
                              int32_t* ids, float* scores, int32_t* ranks, int32_t* counts, void* stream) {
  if (num_rows == 0) return B200KV_OK;
  if (!x || !router_w || !ids || !scores || !ranks || !counts) return B200KV_E_NULL;
  if (num_rows < 0 || width < 1 || experts < 1 || experts > kRtMaxExperts || top < 1 || top > experts) return B200KV_E_SHAPE;
  if (!aligned(x, 16) || !aligned(router_w, 16)) return B200KV_E_ALIGN;
  cudaStream_t s = (cudaStream_t)stream;
  const int groups = (experts + kRtExperts - 1) / kRtExperts;
  const int slices = groups >= kRtWarps ? 1 : kRtWarps / groups;
  const int extra = slices > 1 ? slices : 0;
  const size_t smem1 = (size_t)((width + 3) / 4 * 4 + (1 + extra) * experts) * 4, smem4 = 4 * smem1;
  if (smem1 > 220 * 1024) return B200KV_E_RANGE;
  if (num_rows >= 512 && smem4 <= 72 * 1024) {
    if (cudaFuncSetAttribute(router_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem4) != cudaSuccess) return B200KV_E_LAUNCH;
    return launch_result(launch_chained(router_kernel<4>, dim3((num_rows + 3) / 4), dim3(kRtWarps * 32), smem4, s, x, (const uint16_t*)router_w,
                                        num_rows, width, experts, top, slices, ids, scores, ranks, counts));
  }
  if (cudaFuncSetAttribute(router_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1) != cudaSuccess) return B200KV_E_LAUNCH;
  return launch_result(launch_chained(router_kernel<1>, dim3(num_rows), dim3(kRtWarps * 32), smem1, s, x, (const uint16_t*)router_w, num_rows,
                                      width, experts, top, slices, ids, scores, ranks, counts));
}

extern "C" int b200dec_dispatch(const void* xb, int32_t elem, const int32_t* ids, const float* scores, const int32_t* ranks,
                                const int32_t* counts, int32_t num_rows, int32_t width, int32_t experts, int32_t top, int32_t tile_rows,
                                void* x_sorted, float* score_sorted, int32_t* slots, int32_t* tiles, int32_t max_tiles, void* stream) {
  if (num_rows == 0) return B200KV_OK;
  if (!xb || !ids || !scores || !ranks || !counts || !x_sorted || !score_sorted || !slots || !tiles) return B200KV_E_NULL;
  if (num_rows < 0 || width < 1 || experts < 1 || experts > kRtMaxExperts || top < 1 || tile_rows < 1 || max_tiles < 1 || (elem != 2 && elem != 4))
    return B200KV_E_SHAPE;
  if (!aligned(xb, 16) || !aligned(x_sorted, 16)) return B200KV_E_ALIGN;
  const dim3 grid(num_rows < 148 * 8 ? num_rows : 148 * 8);
  cudaStream_t s = (cudaStream_t)stream;
  if (elem == 2)
    return launch_result(launch_chained(dispatch_kernel<uint16_t>, grid, dim3(kDpThreads), 0, s, (const uint16_t*)xb, ids, scores, ranks, counts,
                                        num_rows, width, experts, top, tile_rows, (uint16_t*)x_sorted, score_sorted, slots, tiles, max_tiles));
  return launch_result(launch_chained(dispatch_kernel<float>, grid, dim3(kDpThreads), 0, s, (const float*)xb, ids, scores, ranks, counts, num_rows,
                                      width, experts, top, tile_rows, (float*)x_sorted, score_sorted, slots, tiles, max_tiles));
}

extern "C" int b200dec_grouped_linear(const void* x, const void* w, int32_t elem, const int32_t* tiles, int32_t max_tiles, int32_t tile_rows,
                                      int32_t total_rows, int32_t experts, int32_t out_rows, int32_t width, const float* score_sorted,
                                      int32_t act, float limit, float slope, void* y, int32_t sm_count, int32_t variant, int32_t* status,
                                      void* stream) {
  if (total_rows == 0) return B200KV_OK;
  if (!x || !w || !tiles || !y || (act && !score_sorted)) return B200KV_E_NULL;
  if (total_rows < 0 || max_tiles < 1 || tile_rows < 1 || experts < 1 || out_rows < 1 || width < 1 || (act && out_rows % 2) ||
      (elem != 2 && elem != 4) || sm_count < 1)
    return B200KV_E_SHAPE;
  if (!aligned(x, 16) || !aligned(w, 16) || !aligned(y, 16)) return B200KV_E_ALIGN;
  cudaStream_t s = (cudaStream_t)stream;
  if (variant == 0) {
    if (elem != 2 || width % 8) return B200KV_E_SHAPE;
    return launch_grouped_linear_tc5(x, w, tiles, max_tiles, tile_rows, total_rows, experts, out_rows, width, score_sorted, act, limit, slope, y,
                                     sm_count, status, s);
  }
  const dim3 grid((out_rows + kGsCols - 1) / kGsCols, max_tiles < 65535 ? max_tiles : 65535);
  if (elem == 2)
    return launch_result(launch_chained(grouped_linear_simt_kernel<uint16_t>, grid, dim3(kGsThreads), 0, s, (const uint16_t*)x, (const uint16_t*)w,
                                        tiles, out_rows, width, score_sorted, act, limit, slope, (uint16_t*)y));
  return launch_result(launch_chained(grouped_linear_simt_kernel<float>, grid, dim3(kGsThreads), 0, s, (const float*)x, (const float*)w, tiles,
                                      out_rows, width, score_sorted, act, limit, slope, (float*)y));
}
