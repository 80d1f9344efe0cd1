// Row-wise ops of a decoder with a 32-bit residual stream: embedding rows, and the residual update of the
// norm-after-the-sum arrangement with the optional sum over a token's experts.  HBM-bound streaming kernels; one
// block per row, the row in registers between the two passes.  Also the arrangement with the norm on a sublayer's output,
// the gated unit of a dense feed-forward, and the norm of a row's parts with a gate.
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

// x += mult * rmsnorm(y) * weight, one block per row.  kChunks > 0: y in registers between the passes (width % 4 == 0),
// 0: any width, y is read twice.
template <typename T, int kChunks>
__global__ void __launch_bounds__(kRowThreads)
norm_add_kernel(float* x, const T* __restrict__ y, const float* __restrict__ weight, float mult, float eps, T* __restrict__ xb, int width) {
  pdl_enter();
  pdl_wait();
  const long long at = (long long)blockIdx.x * width;
  float ss = 0.f;
  if (kChunks > 0) {
    float f[kChunks > 0 ? kChunks : 1][4], old[kChunks > 0 ? kChunks : 1][4];
#pragma unroll
    for (int c = 0; c < kChunks; ++c) {
      const int col = (c * kRowThreads + threadIdx.x) * 4;
      if (col < width) {
        ld_elem4(y + at + col, f[c]);
        ld_fresh4(x + at + col, old[c]);
#pragma unroll
        for (int i = 0; i < 4; ++i) ss = fmaf(f[c][i], f[c][i], ss);
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
        for (int i = 0; i < 4; ++i) f[c][i] = fmaf(mult, f[c][i] * inv * w[i], old[c][i]);
        st_elem4(x + at + col, f[c]);
        if (xb) st_elem4(xb + at + col, f[c]);
      }
    }
  } else {
    for (int c = threadIdx.x; c < width; c += kRowThreads) {
      const float f = ld_elem(y + at + c);
      ss = fmaf(f, f, ss);
    }
    const float inv = 1.0f / sqrtf(row_sum(ss) / (float)width + eps);
    for (int c = threadIdx.x; c < width; c += kRowThreads) {
      const float f = fmaf(mult, ld_elem(y + at + c) * inv * weight[c], ld_fresh(x + at + c));
      x[at + c] = f;
      if (xb) st_elem(xb + at + c, f);
    }
  }
}

// kVec channels (8, or 1 for any size) of one row per thread.
template <typename T, int kVec>
__global__ void __launch_bounds__(kRowThreads)
silu_mul_rows_kernel(const T* __restrict__ gu, long long stride, T* __restrict__ out, long long out_stride, int rows, int ff) {
  pdl_enter();
  pdl_wait();
  const long long r = blockIdx.x;
  const int c = (blockIdx.y * kRowThreads + threadIdx.x) * kVec;
  if (c >= ff) return;
  const T* src = gu + r * stride + c;
  float g[kVec], u[kVec];
  ld_vec(src, g);
  ld_vec(src + ff, u);
#pragma unroll
  for (int e = 0; e < kVec; ++e) g[e] = g[e] * sigmoid_act<T>(g[e]) * u[e];
  st_vec(out + r * out_stride + c, g);
}

// Norm of every part of a row by itself with a gate before or after: kThreads threads per part (a warp or the block), kVec
// neighbouring channels at a time, kKeep such groups in registers per thread (0: read twice).
template <typename T, int kThreads, int kVec, int kKeep>
__global__ void __launch_bounds__(kRowThreads)
gated_norm_kernel(const float* __restrict__ o, const T* __restrict__ gate, long long gate_stride, int gate_first,
                  const float* __restrict__ weight, int weight_len, float eps, float out_scale, T* __restrict__ out, long long out_stride,
                  int rows, int len, int parts) {
  pdl_enter();
  const int part = len / parts;
  const long long item = (long long)blockIdx.x * (kRowThreads / kThreads) + threadIdx.x / kThreads;
  const int t = threadIdx.x % kThreads;
  pdl_wait();
  const int r = (int)(item / parts), p = (int)(item - (long long)r * parts);
  const bool live = r < rows;  // the same for all threads of a part
  const float* src = o + (long long)r * len + p * part;
  const T* g = gate + r * gate_stride + p * part;
  T* dst = out + r * out_stride + p * part;
  // v: the value before the norm, f: what it is multiplied by behind it
  auto load = [&](int c, float (&v)[kVec], float (&f)[kVec]) {
    float z[kVec];
    ld_vec(src + c, v);
    ld_vec(g + c, z);
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      const float s = sigmoid_act<T>(z[i]);
      f[i] = gate_first ? 1.f : s;
      if (gate_first) v[i] *= z[i] * s;
    }
  };
  auto put = [&](int c, float inv, float (&v)[kVec], const float (&f)[kVec]) {
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      const int at = p * part + c + i;
      v[i] = v[i] * inv * weight[weight_len == len ? at : at % weight_len] * f[i] * out_scale;
    }
    st_vec(dst + c, v);
  };
  float v[kKeep > 0 ? kKeep : 1][kVec], f[kKeep > 0 ? kKeep : 1][kVec], ss = 0.f;
  if (live) {
    if (kKeep > 0) {
#pragma unroll
      for (int i = 0; i < kKeep; ++i) {
        const int c = (t + i * kThreads) * kVec;
        if (c < part) {
          load(c, v[i], f[i]);
#pragma unroll
          for (int k = 0; k < kVec; ++k) ss = fmaf(v[i][k], v[i][k], ss);
        }
      }
    } else {
      for (int c = t * kVec; c < part; c += kThreads * kVec) {
        load(c, v[0], f[0]);
#pragma unroll
        for (int k = 0; k < kVec; ++k) ss = fmaf(v[0][k], v[0][k], ss);
      }
    }
  }
  ss = kThreads == 32 ? warp_sum(ss) : row_sum(ss);
  if (!live) return;
  const float inv = 1.0f / sqrtf(ss / (float)part + eps);
  if (kKeep > 0) {
#pragma unroll
    for (int i = 0; i < kKeep; ++i)
      if ((t + i * kThreads) * kVec < part) put((t + i * kThreads) * kVec, inv, v[i], f[i]);
  } else {
    for (int c = t * kVec; c < part; c += kThreads * kVec) {
      load(c, v[0], f[0]);
      put(c, inv, v[0], f[0]);
    }
  }
}

template <typename T>
static int run_norm_add(float* x, const void* y, const float* weight, float mult, float eps, void* xb, int rows, int width, cudaStream_t s) {
  auto* kernel = width % 4 ? norm_add_kernel<T, 0>
                 : width <= kRowThreads * 8 ? norm_add_kernel<T, 2>
                 : width <= kRowThreads * 4 * kRowChunks ? norm_add_kernel<T, kRowChunks> : norm_add_kernel<T, 0>;
  return launch_result(launch_chained(kernel, dim3(rows), dim3(kRowThreads), 0, s, x, (const T*)y, weight, mult, eps, (T*)xb, width));
}

template <typename T>
static int run_gated_norm(const float* o, const void* gate, int64_t gate_stride, int gate_first, const float* weight, int weight_len,
                          float eps, float out_scale, void* out, int64_t out_stride, int rows, int len, int parts,
                          cudaStream_t s) {
  const int part = len / parts;
  const bool vec = part % 4 == 0 && len % 4 == 0 && gate_stride % 4 == 0 && out_stride % 4 == 0 && aligned(o, 16) && aligned(gate, 16) &&
                   aligned(out, 16);
  const bool warp = part <= (vec ? 512 : 256);
  auto* kernel = vec ? (part <= 128   ? gated_norm_kernel<T, 32, 4, 1>
                        : warp        ? gated_norm_kernel<T, 32, 4, 4>
                        : part <= 1024 ? gated_norm_kernel<T, kRowThreads, 4, 1>
                        : part <= 4096 ? gated_norm_kernel<T, kRowThreads, 4, 4>
                                       : gated_norm_kernel<T, kRowThreads, 4, 0>)
                     : (warp ? gated_norm_kernel<T, 32, 1, 8> : gated_norm_kernel<T, kRowThreads, 1, 0>);
  const long long items = (long long)rows * parts, per = warp ? kRowThreads / 32 : 1, blocks = (items + per - 1) / per;
  if (blocks > 0x7FFFFFF0ll) return B200KV_E_RANGE;
  return launch_result(launch_chained(kernel, dim3((unsigned)blocks), dim3(kRowThreads), 0, s, o, (const T*)gate, (long long)gate_stride,
                                      gate_first, weight, weight_len, eps, out_scale, (T*)out, (long long)out_stride, rows, len, parts));
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

extern "C" int b200dec_norm_add(float* x, const void* y, int32_t elem, const float* weight, float mult, float eps, void* xb,
                                int32_t num_rows, int32_t width, void* stream) {
  if (num_rows == 0) return B200KV_OK;
  if (!x || !y || !weight) return B200KV_E_NULL;
  if (num_rows < 0 || width < 1 || (elem != 2 && elem != 4)) return B200KV_E_SHAPE;
  if (!aligned(x, 16) || !aligned(y, 16) || !aligned(weight, 16) || !aligned(xb, 16)) return B200KV_E_ALIGN;
  cudaStream_t s = (cudaStream_t)stream;
  return elem == 2 ? run_norm_add<uint16_t>(x, y, weight, mult, eps, xb, num_rows, width, s)
                   : run_norm_add<float>(x, y, weight, mult, eps, xb, num_rows, width, s);
}

extern "C" int b200dec_silu_mul(const void* gate_up, int64_t stride, int32_t elem, void* out, int64_t out_stride, int32_t num_rows,
                                int32_t ff, void* stream) {
  if (num_rows == 0) return B200KV_OK;
  if (!gate_up || !out) return B200KV_E_NULL;
  if (num_rows < 0 || ff < 1 || stride < 2 * (int64_t)ff || out_stride < ff || (elem != 2 && elem != 4)) return B200KV_E_SHAPE;
  const bool vec = ff % 8 == 0 && stride % 8 == 0 && out_stride % 8 == 0 && aligned(gate_up, 16) && aligned(out, 16);
  const dim3 grid(num_rows, (ff / (vec ? 8 : 1) + kRowThreads - 1) / kRowThreads);
  cudaStream_t s = (cudaStream_t)stream;
  if (elem == 2)
    return launch_result(launch_chained(vec ? silu_mul_rows_kernel<uint16_t, 8> : silu_mul_rows_kernel<uint16_t, 1>, grid, dim3(kRowThreads), 0, s,
                                        (const uint16_t*)gate_up, (long long)stride, (uint16_t*)out, (long long)out_stride, num_rows, ff));
  return launch_result(launch_chained(vec ? silu_mul_rows_kernel<float, 8> : silu_mul_rows_kernel<float, 1>, grid, dim3(kRowThreads), 0, s,
                                      (const float*)gate_up, (long long)stride, (float*)out, (long long)out_stride, num_rows, ff));
}

extern "C" int b200dec_gated_norm(const float* o, const void* gate, int64_t gate_stride, int32_t gate_first, int32_t elem,
                                  const float* weight, int32_t weight_len, float eps, float out_scale, void* out, int64_t out_stride,
                                  int32_t num_rows, int32_t len, int32_t parts, void* stream) {
  if (num_rows == 0) return B200KV_OK;
  if (!o || !gate || !weight || !out) return B200KV_E_NULL;
  if (num_rows < 0 || len < 1 || parts < 1 || len % parts || weight_len < 1 || len % weight_len || (elem != 2 && elem != 4))
    return B200KV_E_SHAPE;
  cudaStream_t s = (cudaStream_t)stream;
  return elem == 2 ? run_gated_norm<uint16_t>(o, gate, gate_stride, gate_first, weight, weight_len, eps, out_scale, out, out_stride,
                                              num_rows, len, parts, s)
                   : run_gated_norm<float>(o, gate, gate_stride, gate_first, weight, weight_len, eps, out_scale, out, out_stride, num_rows,
                                           len, parts, s);
}
