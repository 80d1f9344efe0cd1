// Helpers shared by the b200dec kernels: element conversion, cache addressing, reductions.
#pragma once
#include "b200dec.h"
#include "common.cuh"

namespace b200kv {

__device__ __forceinline__ float ld_elem(const uint16_t* p) { return bf16_bits_to_float(*p); }
__device__ __forceinline__ float ld_elem(const float* p) { return *p; }
__device__ __forceinline__ void st_elem(uint16_t* p, float v) { *p = (uint16_t)float_to_bf16_bits(v); }
__device__ __forceinline__ void st_elem(float* p, float v) { *p = v; }

// 4 consecutive elements (16-byte aligned fp32, 8-byte aligned bf16)
__device__ __forceinline__ void ld_elem4(const float* p, float (&f)[4]) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
__device__ __forceinline__ void ld_elem4(const uint16_t* p, float (&f)[4]) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xFFFF0000u);
  f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xFFFF0000u);
}
// The same through L2 only.  With chained launches a kernel is brought up while the one before it still runs, so its
// multiprocessor's L1 may hold a line that the predecessor read before another of its blocks wrote part of it.  Whatever the
// predecessor produces next to (or over) what it reads is therefore loaded this way.
__device__ __forceinline__ void ld_fresh4(const float* p, float (&f)[4]) {
  const float4 v = __ldcg(reinterpret_cast<const float4*>(p));
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
__device__ __forceinline__ float ld_fresh(const float* p) { return __ldcg(p); }
__device__ __forceinline__ int ld_fresh(const int32_t* p) { return __ldcg(p); }

__device__ __forceinline__ void st_elem4(float* p, const float (&f)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
__device__ __forceinline__ void st_elem4(uint16_t* p, const float (&f)[4]) {
  uint2 v;
  v.x = float_to_bf16_bits(f[0]) | (float_to_bf16_bits(f[1]) << 16);
  v.y = float_to_bf16_bits(f[2]) | (float_to_bf16_bits(f[3]) << 16);
  *reinterpret_cast<uint2*>(p) = v;
}

// kVec consecutive elements (aligned to their size; 8 bf16 in one 16-byte access)
__device__ __forceinline__ void ld_vec(const uint16_t* p, float (&f)[1]) { f[0] = ld_elem(p); }
__device__ __forceinline__ void ld_vec(const float* p, float (&f)[1]) { f[0] = *p; }
__device__ __forceinline__ void ld_vec(const uint16_t* p, float (&f)[4]) { ld_elem4(p, f); }
__device__ __forceinline__ void ld_vec(const float* p, float (&f)[4]) { ld_elem4(p, f); }
__device__ __forceinline__ void unpack8(const uint4& v, float (&f)[8]) {
  f[0] = __uint_as_float(v.x << 16); f[1] = __uint_as_float(v.x & 0xFFFF0000u);
  f[2] = __uint_as_float(v.y << 16); f[3] = __uint_as_float(v.y & 0xFFFF0000u);
  f[4] = __uint_as_float(v.z << 16); f[5] = __uint_as_float(v.z & 0xFFFF0000u);
  f[6] = __uint_as_float(v.w << 16); f[7] = __uint_as_float(v.w & 0xFFFF0000u);
}
__device__ __forceinline__ void ld_vec(const uint16_t* p, float (&f)[8]) { unpack8(*reinterpret_cast<const uint4*>(p), f); }
__device__ __forceinline__ void ld_vec(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void st_vec(uint16_t* p, const float (&f)[1]) { st_elem(p, f[0]); }
__device__ __forceinline__ void st_vec(float* p, const float (&f)[1]) { *p = f[0]; }
__device__ __forceinline__ void st_vec(uint16_t* p, const float (&f)[4]) { st_elem4(p, f); }
__device__ __forceinline__ void st_vec(float* p, const float (&f)[4]) { st_elem4(p, f); }
__device__ __forceinline__ void st_vec(uint16_t* p, const float (&f)[8]) {
  uint4 v;
  v.x = float_to_bf16_bits(f[0]) | (float_to_bf16_bits(f[1]) << 16);
  v.y = float_to_bf16_bits(f[2]) | (float_to_bf16_bits(f[3]) << 16);
  v.z = float_to_bf16_bits(f[4]) | (float_to_bf16_bits(f[5]) << 16);
  v.w = float_to_bf16_bits(f[6]) | (float_to_bf16_bits(f[7]) << 16);
  *reinterpret_cast<uint4*>(p) = v;
}
__device__ __forceinline__ void st_vec(float* p, const float (&f)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// Device view of a b200dec_cache with its page table.
struct DecCache {
  void* k;
  void* v;
  int num_pages, heads, P, k_dim, v_dim, k_row, v_row;
  const int32_t* table;
  int table_stride, max_pages;
};
inline DecCache dec_view(const b200dec_cache* c, const b200kv_table* t) {
  return DecCache{c->k, c->v, c->num_pages, c->kv_heads, c->page_size, c->k_dim, c->v_dim, c->k_row, c->v_row,
                  t->ids, t->stride, t->max_pages};
}
// Page of token position `pos` of entry b, or -1 (with a status bit).
__device__ __forceinline__ int dec_page(const DecCache& c, int b, int pos, int32_t* status) {
  const int slot = pos / c.P;
  if (pos < 0 || slot >= c.max_pages) {
    if (status) atomicOr(status, B200KV_S_BAD_POSITION);
    return -1;
  }
  const int page = c.table[(long long)b * c.table_stride + slot];
  if (page < 0 || page >= c.num_pages) {
    if (status) atomicOr(status, B200KV_S_BAD_PAGE);
    return -1;
  }
  return page;
}
// First element of row `prow` of (page, head) in k / v.
__device__ __forceinline__ long long dec_row(const DecCache& c, int page, int head, int prow) {
  return ((long long)page * c.heads + head) * c.P + prow;
}

inline int check_dec_cache(const b200dec_cache* c, const b200kv_table* t) {
  if (!c || !t || !c->k || !c->v || !t->ids) return B200KV_E_NULL;
  if (c->num_pages < 1 || c->kv_heads < 1 || c->page_size < 1 || c->k_dim < 1 || c->v_dim < 1) return B200KV_E_SHAPE;
  if (c->k_row != (c->k_dim + 7) / 8 * 8 || c->v_row != (c->v_dim + 7) / 8 * 8) return B200KV_E_SHAPE;
  if (c->elem != 2 && c->elem != 4) return B200KV_E_SHAPE;
  if (t->max_pages < 1 || t->stride < 0) return B200KV_E_SHAPE;
  if (!aligned(c->k, 16) || !aligned(c->v, 16)) return B200KV_E_ALIGN;
  return B200KV_OK;
}

// sigmoid of an activation or output gate: in a bf16 model by the hardware's exponential and division (a few units of the
// last 32-bit place), far below the bf16 rounding of what it multiplies
template <typename T>
__device__ __forceinline__ float sigmoid_act(float z) {
  if constexpr (sizeof(T) == 4) return sigmoid_f(z);
  else return __fdividef(1.f, 1.f + __expf(-fmaxf(z, -80.f)));  // the quotient is defined up to 2^126
}

// Device view of b200dec_attn_options (defaults filled in).
struct DecAttnOpt {
  int window;
  const float* sink;
  const void* gate;
  long long gate_stride, out_stride;
  float out_scale;
  // what the finished output of (row, head) is multiplied by
  template <typename T>
  __device__ __forceinline__ float factor(long long r, int h) const {
    return gate ? out_scale * sigmoid_f(ld_elem((const T*)gate + r * gate_stride + h)) : out_scale;
  }
};
inline int dec_attn_opt(const b200dec_attn_options* o, int heads, int v_dim, DecAttnOpt* d) {
  *d = DecAttnOpt{0, nullptr, nullptr, 0, (long long)heads * v_dim, 1.f};
  if (!o) return B200KV_OK;
  d->window = o->window;
  d->sink = o->sink;
  d->gate = o->gate;
  d->gate_stride = o->gate_stride;
  d->out_scale = o->out_scale;
  if (o->window < 0) return B200KV_E_SHAPE;
  if (o->out_stride) {
    if (o->out_stride < d->out_stride || o->out_stride % 8) return B200KV_E_SHAPE;
    d->out_stride = o->out_stride;
  }
  return B200KV_OK;
}

inline int launch_result(cudaError_t e) { return e == cudaSuccess && cudaGetLastError() == cudaSuccess ? B200KV_OK : B200KV_E_LAUNCH; }

}  // namespace b200kv
