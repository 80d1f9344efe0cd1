// Row-wise ops of a decoder with a 32-bit residual stream: embedding rows, and the residual update of the
// norm-after-the-sum arrangement with the optional sum over a token's experts.  HBM-bound streaming kernels; one
// block per row, the row in registers between the two passes.
#include "dec_common.cuh"

namespace b200kv {

constexpr int kRowThreads = 256;
constexpr int kRowChunks = 8;  // the register path holds rows of up to 256 * 4 * 8 = 8192 channels (2 chunks: 2048)

__device__ __forceinline__ float row_sum(float v) {
  __shared__ float part[kRowThreads / 32];
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int i = 0; i < kRowThreads / 32; ++i) tot += part[i];
  return tot;
}

template <typename T>
__global__ void __launch_bounds__(kRowThreads)
embed_kernel(const T* __restrict__ table, const int32_t* __restrict__ ids, float* __restrict__ x, T* __restrict__ xb, int width,
             int vocab, int32_t* status) {
  pdl_enter();
  const long long r = blockIdx.x;
  int id = ids[r];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0 && status) atomicOr(status, B200KV_S_BAD_POSITION);
    id = 0;
  }
  pdl_wait();
  const T* src = table + (long long)id * width;
  if (width % 4 == 0) {
    for (int c = threadIdx.x * 4; c < width; c += kRowThreads * 4) {
      float f[4];
      ld_elem4(src + c, f);
      st_elem4(x + r * width + c, f);
      if (xb) st_elem4(xb + r * width + c, f);
    }
  } else {
    for (int c = threadIdx.x; c < width; c += kRowThreads) {
      const float f = ld_elem(src + c);
      x[r * width + c] = f;
      if (xb) xb[r * width + c] = src[c];
    }
  }
}

// The registers path: width % 4 == 0 and width <= 8192.
template <typename T, int kChunks>
__global__ void __launch_bounds__(kRowThreads)
scaled_add_norm_kernel(const float* x, const T* __restrict__ delta, const int32_t* __restrict__ index, int top,
                       const float* __restrict__ weight, float alpha, float eps, float* x_out, T* __restrict__ xb_out,
                       int width, int32_t* __restrict__ zero, int num_zero) {
  pdl_enter();
  pdl_wait();
  const long long r = blockIdx.x;
  if (zero && blockIdx.x == 0)
    for (int i = threadIdx.x; i < num_zero; i += kRowThreads) zero[i] = 0;
  float s[kChunks][4];
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int col = (c * kRowThreads + threadIdx.x) * 4;
    if (col < width) {
      ld_fresh4(x + r * width + col, s[c]);
#pragma unroll
      for (int i = 0; i < 4; ++i) s[c][i] *= alpha;
      if (delta) {
        for (int j = 0; j < top; ++j) {
          const long long row = index ? ld_fresh(index + r * top + j) : r;
          float d[4];
          ld_elem4(delta + row * width + col, d);
#pragma unroll
          for (int i = 0; i < 4; ++i) s[c][i] += d[i];
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) ss = fmaf(s[c][i], s[c][i], ss);
    }
  }
  const float inv = 1.0f / sqrtf(row_sum(ss) / (float)width + eps);
#pragma unroll
  for (int c = 0; c < kChunks; ++c) {
    const int col = (c * kRowThreads + threadIdx.x) * 4;
    if (col < width) {
      float w[4];
      ld_elem4(weight + col, w);
#pragma unroll
      for (int i = 0; i < 4; ++i) s[c][i] = s[c][i] * inv * w[i];
      if (x_out) st_elem4(x_out + r * width + col, s[c]);
      if (xb_out) st_elem4(xb_out + r * width + col, s[c]);
    }
  }
}

// Any width: the sums are kept in dynamic shared memory.
template <typename T>
__global__ void __launch_bounds__(kRowThreads)
scaled_add_norm_any_kernel(const float* x, const T* __restrict__ delta, const int32_t* __restrict__ index, int top,
                           const float* __restrict__ weight, float alpha, float eps, float* x_out,
                           T* __restrict__ xb_out, int width, int32_t* __restrict__ zero, int num_zero) {
  extern __shared__ float srow[];
  pdl_enter();
  pdl_wait();
  const long long r = blockIdx.x;
  if (zero && blockIdx.x == 0)
    for (int i = threadIdx.x; i < num_zero; i += kRowThreads) zero[i] = 0;
  float ss = 0.f;
  for (int c = threadIdx.x; c < width; c += kRowThreads) {
    float s = alpha * ld_fresh(x + r * width + c);
    if (delta)
      for (int j = 0; j < top; ++j) s += ld_elem(delta + (index ? (long long)ld_fresh(index + r * top + j) : r) * width + c);
    srow[c] = s;
    ss = fmaf(s, s, ss);
  }
  const float inv = 1.0f / sqrtf(row_sum(ss) / (float)width + eps);
  for (int c = threadIdx.x; c < width; c += kRowThreads) {
    const float y = srow[c] * inv * weight[c];
    if (x_out) x_out[r * width + c] = y;
    if (xb_out) st_elem(xb_out + r * width + c, y);
  }
}

template <typename T>
static int run_scaled_add_norm(const float* x, const void* delta, const int32_t* index, int top, const float* weight, float alpha,
                               float eps, float* x_out, void* xb_out, int rows, int width, int32_t* zero, int num_zero,
                               cudaStream_t stream) {
  if (width % 4 == 0 && width <= kRowThreads * 4 * 2)
    return launch_result(launch_chained(scaled_add_norm_kernel<T, 2>, dim3(rows), dim3(kRowThreads), 0, stream, x, (const T*)delta, index,
                                        top, weight, alpha, eps, x_out, (T*)xb_out, width, zero, num_zero));
  if (width % 4 == 0 && width <= kRowThreads * 4 * kRowChunks)
    return launch_result(launch_chained(scaled_add_norm_kernel<T, kRowChunks>, dim3(rows), dim3(kRowThreads), 0, stream, x, (const T*)delta, index,
                                        top, weight, alpha, eps, x_out, (T*)xb_out, width, zero, num_zero));
  const size_t smem = (size_t)width * 4;
  if (smem > 200 * 1024) return B200KV_E_RANGE;
  if (cudaFuncSetAttribute(scaled_add_norm_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return B200KV_E_LAUNCH;
  return launch_result(launch_chained(scaled_add_norm_any_kernel<T>, dim3(rows), dim3(kRowThreads), smem, stream, x, (const T*)delta,
                                      index, top, weight, alpha, eps, x_out, (T*)xb_out, width, zero, num_zero));
}

}  // namespace b200kv

using namespace b200kv;

extern "C" int b200dec_embed(const void* table, int32_t elem, const int32_t* ids, float* x, void* xb, int32_t num_rows,
                             int32_t width, int32_t vocab, int32_t* status, void* stream) {
  if (num_rows == 0) return B200KV_OK;
  if (!table || !ids || !x) return B200KV_E_NULL;
  if (num_rows < 0 || width < 1 || vocab < 1 || (elem != 2 && elem != 4)) return B200KV_E_SHAPE;
  if (!aligned(table, 16) || !aligned(x, 16) || !aligned(xb, 16)) return B200KV_E_ALIGN;
  cudaStream_t s = (cudaStream_t)stream;
  if (elem == 2)
    return launch_result(launch_chained(embed_kernel<uint16_t>, dim3(num_rows), dim3(kRowThreads), 0, s, (const uint16_t*)table, ids, x,
                                        (uint16_t*)xb, width, vocab, status));
  return launch_result(launch_chained(embed_kernel<float>, dim3(num_rows), dim3(kRowThreads), 0, s, (const float*)table, ids, x,
                                      (float*)xb, width, vocab, status));
}

extern "C" int b200dec_scaled_add_norm(const float* x, const void* delta, const int32_t* index, int32_t top, int32_t elem,
                                       const float* weight, float alpha, float eps, float* x_out, void* xb_out, int32_t num_rows,
                                       int32_t width, int32_t* zero, int32_t num_zero, void* stream) {
  if (num_rows == 0) return B200KV_OK;
  if (!x || !weight) return B200KV_E_NULL;
  if (num_rows < 0 || width < 1 || top < 1 || (!index && top != 1) || (elem != 2 && elem != 4)) return B200KV_E_SHAPE;
  if (!aligned(x, 16) || !aligned(delta, 16) || !aligned(weight, 16) || !aligned(x_out, 16) || !aligned(xb_out, 16))
    return B200KV_E_ALIGN;
  cudaStream_t s = (cudaStream_t)stream;
  if (elem == 2)
    return run_scaled_add_norm<uint16_t>(x, delta, index, top, weight, alpha, eps, x_out, xb_out, num_rows, width, zero, num_zero, s);
  return run_scaled_add_norm<float>(x, delta, index, top, weight, alpha, eps, x_out, xb_out, num_rows, width, zero, num_zero, s);
}
