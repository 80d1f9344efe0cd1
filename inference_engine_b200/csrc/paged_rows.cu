// The paged cache of unquantised rows: rotary positions + unit norm + write of keys and values (one kernel; a second one
// norms whole projections first and rotates neighbouring channels), and the
// general attention over it (any sizes, bf16 or fp32, prompt portions and decoding alike) on the CUDA cores.
#include "dec_common.cuh"

namespace b200kv {

constexpr int kRwWarps = 8;
constexpr int kRwMaxPairs = 16;  // a lane holds up to 32 channels: heads of up to 1024 (2: heads of up to 128)

__device__ __forceinline__ float2 rw_load2(const uint16_t* p) {
  const uint32_t u = *reinterpret_cast<const uint32_t*>(p);
  return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xFFFF0000u));
}
__device__ __forceinline__ float2 rw_load2(const float* p) { return *reinterpret_cast<const float2*>(p); }

// One warp per (row, head), heads in the order q | k | v.  A lane owns channels 2 * lane + 64 * i and the next one.
// kPairs: head sizes, half and the row stride are even, so both channels are loaded and rotated together.
template <typename T, bool kPairs, int kMax>
__global__ void __launch_bounds__(kRwWarps * 32)
rope_write_kernel(const T* __restrict__ qkv, long long qkv_stride, b200dec_rows rows, DecCache c, const float* __restrict__ cos_sin,
                  int table_len, int half, int heads, int write_kv, int unit_norm, float eps, T* __restrict__ q_out, int32_t* status) {
  pdl_enter();
  const int hkv = write_kv ? c.heads : 0, per_row = heads + 2 * hkv;
  const int item = blockIdx.x * kRwWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (item >= rows.num_rows * per_row) return;
  const int r = item / per_row, j = item - r * per_row;
  const int kind = j < heads ? 0 : (j < heads + hkv ? 1 : 2);  // q, k, v
  int seq = r, pos;
  if (rows.seq_ids) {
    seq = rows.seq_ids[r];
    pos = rows.positions[r];
  } else {
    if (r >= *rows.num_decoding) {  // an idle row: nothing is written to the cache, q reads as zero
      pdl_wait();
      if (kind == 0)
        for (int ch = lane; ch < c.k_row; ch += 32) st_elem(q_out + ((long long)r * heads + j) * c.k_row + ch, 0.f);
      return;
    }
    pos = rows.cached_lens[r];
  }
  const bool ok = pos >= 0 && (half == 0 || pos < table_len);
  if (!ok) {
    if (lane == 0 && status) atomicOr(status, B200KV_S_BAD_POSITION);
    pos = 0;
  }
  T* dst;
  int dim = c.k_dim, row_len = c.k_row;
  long long src_off;
  if (kind == 0) {
    dst = q_out + ((long long)r * heads + j) * c.k_row;
    src_off = (long long)j * c.k_dim;
  } else {
    const int h = kind == 1 ? j - heads : j - heads - hkv;
    const int page = ok ? dec_page(c, seq, pos, lane == 0 ? status : nullptr) : -1;
    if (page < 0) return;
    const long long at = dec_row(c, page, h, pos % c.P);
    if (kind == 1) {
      dst = (T*)c.k + at * c.k_row;
      src_off = (long long)(heads + h) * c.k_dim;
    } else {
      dst = (T*)c.v + at * c.v_row;
      src_off = (long long)(heads + hkv) * c.k_dim + (long long)h * c.v_dim;
      dim = c.v_dim;
      row_len = c.v_row;
    }
  }
  pdl_wait();
  const T* src = qkv + r * qkv_stride + src_off;
  float y[kMax][2];
  float ss = 0.f;
  const float2* cs = reinterpret_cast<const float2*>(cos_sin) + (long long)pos * half;
#pragma unroll
  for (int i = 0; i < kMax; ++i) {
    y[i][0] = y[i][1] = 0.f;
    if (kPairs && 64 * i < dim) {
      const int ch = 64 * i + 2 * lane;
      if (ch < dim) {
        float2 v = rw_load2(src + ch);
        if (kind < 2 && ch < 2 * half) {
          const bool low = ch < half;
          const float2 other = rw_load2(src + (low ? ch + half : ch - half));
          const float4 a = *reinterpret_cast<const float4*>(cs + (low ? ch : ch - half));  // cos, sin of both
          const float s0 = low ? -a.y : a.y, s1 = low ? -a.w : a.w;
          v = make_float2(v.x * a.x + other.x * s0, v.y * a.z + other.y * s1);
        }
        y[i][0] = v.x;
        y[i][1] = v.y;
        ss = fmaf(v.x, v.x, fmaf(v.y, v.y, ss));
      }
    } else if (64 * i < dim) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int ch = 64 * i + 2 * lane + e;
        float v = 0.f;
        if (ch < dim) {
          v = ld_elem(src + ch);
          if (kind < 2 && ch < 2 * half) {
            const bool low = ch < half;
            const float other = ld_elem(src + (low ? ch + half : ch - half));
            const float2 a = cs[low ? ch : ch - half];
            v = low ? v * a.x - other * a.y : v * a.x + other * a.y;
          }
        }
        y[i][e] = v;
        ss = fmaf(v, v, ss);
      }
    }
  }
  float inv = 1.f;
  if (kind < 2 && unit_norm) inv = 1.0f / sqrtf(warp_sum(ss) / (float)dim + eps);
#pragma unroll
  for (int i = 0; i < kMax; ++i) {
    const int ch = 64 * i + 2 * lane;
    if (ch < row_len) {  // row_len is even; channels behind dim are zero
      if (sizeof(T) == 2)
        *reinterpret_cast<uint32_t*>(dst + ch) = float_to_bf16_bits(y[i][0] * inv) | (float_to_bf16_bits(y[i][1] * inv) << 16);
      else
        *reinterpret_cast<float2*>(dst + ch) = make_float2(y[i][0] * inv, y[i][1] * inv);
    }
  }
}

// ---------------------------------------------------------------- norm of whole projections, interleaved rotation, write
// One block per row; a thread owns channel pairs tid, tid + 256, ... of q | k | v.
constexpr int kNrThreads = 256;

// Pair p of a group of heads of `pairs` pairs each (shift: log2 of it, or -1).
__device__ __forceinline__ void nr_split(int p, int pairs, int shift, int& head, int& pr) {
  head = shift >= 0 ? p >> shift : p / pairs;
  pr = p - head * pairs;
}

// kKeep > 0: sizes and the row stride are even and a row has at most kKeep * 256 pairs, which stay in registers; their
// weights and angles are loaded beside them.  0: any sizes, the row is read twice.
template <typename T, int kKeep>
__global__ void __launch_bounds__(kNrThreads)
norm_rope_write_kernel(const T* __restrict__ qkv, long long qkv_stride, b200dec_rows rows, DecCache c, const float* __restrict__ q_norm,
                       const float* __restrict__ k_norm, float eps, const float* __restrict__ cos_sin, int table_len, int half, int heads,
                       int k_shift, int v_shift, T* __restrict__ q_out, int32_t* status) {
  __shared__ float part[2][kNrThreads / 32];
  pdl_enter();
  const int r = blockIdx.x, tid = threadIdx.x;
  T* qdst = q_out + (long long)r * heads * c.k_row;
  int seq = r, pos;
  if (rows.seq_ids) {
    seq = rows.seq_ids[r];
    pos = rows.positions[r];
  } else {
    if (r >= *rows.num_decoding) {  // an idle row: nothing is written to the cache, q reads as zero
      pdl_wait();
      for (int ch = tid; ch < heads * c.k_row; ch += kNrThreads) st_elem(qdst + ch, 0.f);
      return;
    }
    pos = rows.cached_lens[r];
  }
  const bool ok = pos >= 0 && (half == 0 || pos < table_len);
  if (!ok) {
    if (tid == 0 && status) atomicOr(status, B200KV_S_BAD_POSITION);
    pos = 0;
  }
  const int page = ok ? dec_page(c, seq, pos, tid == 0 ? status : nullptr) : -1;
  const float2* cs = reinterpret_cast<const float2*>(cos_sin) + (long long)pos * half;
  const T* src = qkv + r * qkv_stride;
  const int nq = heads * c.k_dim, nk = c.heads * c.k_dim, all_heads = heads + c.heads;
  const long long at0 = page < 0 ? 0 : dec_row(c, page, 0, pos % c.P);
  auto put2 = [](T* dst, float a, float b) {
    if (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(dst) = float_to_bf16_bits(a) | (float_to_bf16_bits(b) << 16);
    else *reinterpret_cast<float2*>(dst) = make_float2(a, b);
  };
  // where channel ch of q / k head h (q heads first) goes; only for k heads a page is needed
  auto place = [&](int h, int ch) {
    return h < heads ? qdst + h * c.k_row + ch : (T*)c.k + (at0 + (long long)(h - heads) * c.P) * c.k_row + ch;
  };
  float sq = 0.f, sk = 0.f;
  auto means = [&] {
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if ((tid & 31) == 0) {
      part[0][tid >> 5] = sq;
      part[1][tid >> 5] = sk;
    }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int i = 0; i < kNrThreads / 32; ++i) {
      sq += part[0][i];
      sk += part[1][i];
    }
    sq = 1.0f / sqrtf(sq / (float)nq + eps);
    sk = 1.0f / sqrtf(sk / (float)nk + eps);
  };
  if constexpr (kKeep > 0) {
    const int qkp = (nq + nk) / 2, all = qkp + c.heads * c.v_dim / 2;
    float2 v[kKeep], w[kKeep], t[kKeep];
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {  // nothing here waits for the kernel in front
      const int p = tid + i * kNrThreads;
      if (p < qkp) {
        int h, pr;
        nr_split(p, c.k_dim / 2, k_shift, h, pr);
        w[i] = *reinterpret_cast<const float2*>(2 * p < nq ? q_norm + 2 * p : k_norm + (2 * p - nq));
        t[i] = pr < half ? cs[pr] : make_float2(1.f, 0.f);
      }
    }
    pdl_wait();
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int p = tid + i * kNrThreads;
      if (p < all) v[i] = rw_load2(src + 2 * p);
    }
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int p = tid + i * kNrThreads;
      if (p < qkp) {
        const float s2 = fmaf(v[i].x, v[i].x, v[i].y * v[i].y);
        if (2 * p < nq) sq += s2; else sk += s2;
      }
    }
    means();
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
      const int p = tid + i * kNrThreads;
      int h, pr;
      if (p < qkp) {
        nr_split(p, c.k_dim / 2, k_shift, h, pr);
        if (h >= heads && page < 0) continue;
        const float inv = h < heads ? sq : sk, a = v[i].x * inv * w[i].x, b = v[i].y * inv * w[i].y;
        put2(place(h, 2 * pr), a * t[i].x - b * t[i].y, b * t[i].x + a * t[i].y);
      } else if (p < all && page >= 0) {
        nr_split(p - qkp, c.v_dim / 2, v_shift, h, pr);
        put2((T*)c.v + (at0 + (long long)h * c.P) * c.v_row + 2 * pr, v[i].x, v[i].y);
      }
    }
    // channels behind a size are written as zero
    const int k_pad = (c.k_row - c.k_dim) / 2, v_pad = (c.v_row - c.v_dim) / 2;
    for (int i = tid; i < all_heads * k_pad; i += kNrThreads)
      if (i / k_pad < heads || page >= 0) put2(place(i / k_pad, c.k_dim + 2 * (i % k_pad)), 0.f, 0.f);
    if (page >= 0)
      for (int i = tid; i < c.heads * v_pad; i += kNrThreads)
        put2((T*)c.v + (at0 + (long long)(i / v_pad) * c.P) * c.v_row + c.v_dim + 2 * (i % v_pad), 0.f, 0.f);
  } else {
    pdl_wait();
    for (int i = tid; i < nq + nk; i += kNrThreads) {
      const float f = ld_elem(src + i);
      if (i < nq) sq = fmaf(f, f, sq); else sk = fmaf(f, f, sk);
    }
    means();
    for (int i = tid; i < all_heads * (c.k_row / 2); i += kNrThreads) {
      const int h = i / (c.k_row / 2), pr = i - h * (c.k_row / 2), ch = 2 * pr, off = h * c.k_dim + ch;  // q and k heads lie end to end
      if (h >= heads && page < 0) continue;
      const float* w = h < heads ? q_norm + off : k_norm + (off - nq);
      const float inv = h < heads ? sq : sk;
      float a = ch < c.k_dim ? ld_elem(src + off) * inv * w[0] : 0.f;
      float b = ch + 1 < c.k_dim ? ld_elem(src + off + 1) * inv * w[1] : 0.f;
      if (pr < half) {
        const float2 t = cs[pr];
        const float u = a;
        a = u * t.x - b * t.y;
        b = b * t.x + u * t.y;
      }
      put2(place(h, ch), a, b);
    }
    if (page < 0) return;
    for (int i = tid; i < c.heads * (c.v_row / 2); i += kNrThreads) {
      const int h = i / (c.v_row / 2), ch = 2 * (i - h * (c.v_row / 2));
      const T* p = src + nq + nk + h * c.v_dim + ch;
      put2((T*)c.v + (at0 + (long long)h * c.P) * c.v_row + ch, ch < c.v_dim ? ld_elem(p) : 0.f, ch + 1 < c.v_dim ? ld_elem(p + 1) : 0.f);
    }
  }
}

// ---------------------------------------------------------------- attention, one block per (row, query head)
constexpr int kArThreads = 128;
constexpr int kArKeys = 128;  // keys per block step, one score per thread
constexpr int kArPieces = 8;  // channels of the output per thread: v_dim up to 1024

template <typename T>
__global__ void __launch_bounds__(kArThreads)
attn_rows_kernel(const T* __restrict__ q, DecCache c, b200dec_rows rows, int heads, float scale, DecAttnOpt opt, T* __restrict__ out,
                 int32_t* status) {
  extern __shared__ float ar_smem[];
  float* qs = ar_smem;                                                  // [k_dim]
  float* ps = qs + ((c.k_dim + 3) / 4) * 4;                             // [kArKeys]
  int* pages = reinterpret_cast<int*>(ps + kArKeys);                    // [kArKeys] row index of each key in the cache
  __shared__ float red[2][kArThreads / 32];
  pdl_enter();
  const int r = blockIdx.y, h = blockIdx.x, hk = h / (heads / c.heads), tid = threadIdx.x;
  T* dst = out + r * opt.out_stride + h * c.v_dim;
  int seq = r, pos;
  if (rows.seq_ids) {
    seq = rows.seq_ids[r];
    pos = rows.positions[r];
  } else {
    pos = r < *rows.num_decoding ? rows.cached_lens[r] : -1;
  }
  pdl_wait();
  if (pos < 0) {  // idle row
    for (int ch = tid; ch < c.v_dim; ch += kArThreads) st_elem(dst + ch, 0.f);
    return;
  }
  const T* qrow = q + ((long long)r * heads + h) * c.k_row;
  for (int ch = tid; ch < c.k_dim; ch += kArThreads) qs[ch] = ld_elem(qrow + ch) * scale;
  float m = opt.sink ? opt.sink[h] : -INFINITY, l = opt.sink ? 1.f : 0.f, o[kArPieces];
#pragma unroll
  for (int i = 0; i < kArPieces; ++i) o[i] = 0.f;
  for (int j0 = opt.window > 0 ? max(0, pos - opt.window + 1) : 0; j0 <= pos; j0 += kArKeys) {
    const int n = min(kArKeys, pos + 1 - j0);
    __syncthreads();
    int at = -1;
    float s = -INFINITY;
    if (tid < n) {
      const int page = dec_page(c, seq, j0 + tid, status);
      if (page >= 0) {
        at = page * c.P + (j0 + tid) % c.P;  // token slot; head and row strides are applied below
        const T* krow = (const T*)c.k + dec_row(c, page, hk, (j0 + tid) % c.P) * c.k_row;
        float acc = 0.f;
        for (int ch = 0; ch < c.k_row; ch += 4) {
          float f[4];
          ld_elem4(krow + ch, f);
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (ch + e < c.k_dim) acc = fmaf(qs[ch + e], f[e], acc);
        }
        s = acc;
      }
    }
    pages[tid] = at;
    float mx = s;
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    if ((tid & 31) == 0) red[0][tid >> 5] = mx;
    __syncthreads();
    mx = fmaxf(fmaxf(red[0][0], red[0][1]), fmaxf(red[0][2], red[0][3]));
    const float mn = fmaxf(m, mx), base = mn == -INFINITY ? 0.f : mn;
    const float p = expf(s - base), alpha = expf(m - base);
    m = mn;
    ps[tid] = p;
    const float sum = warp_sum(p);
    if ((tid & 31) == 0) red[1][tid >> 5] = sum;
    __syncthreads();
    l = l * alpha + (red[1][0] + red[1][1]) + (red[1][2] + red[1][3]);
#pragma unroll
    for (int i = 0; i < kArPieces; ++i) o[i] *= alpha;
    for (int k = 0; k < n; ++k) {
      const int slot = pages[k];
      if (slot < 0) continue;
      const int page = slot / c.P;
      const T* vrow = (const T*)c.v + dec_row(c, page, hk, slot - page * c.P) * c.v_row;
      const float w = ps[k];
#pragma unroll
      for (int i = 0; i < kArPieces; ++i) {
        const int ch = tid + i * kArThreads;
        if (ch < c.v_dim) o[i] = fmaf(w, ld_elem(vrow + ch), o[i]);
      }
    }
  }
  const float inv = (l > 0.f ? 1.f / l : 0.f) * opt.factor<T>(r, h);
#pragma unroll
  for (int i = 0; i < kArPieces; ++i) {
    const int ch = tid + i * kArThreads;
    if (ch < c.v_dim) st_elem(dst + ch, o[i] * inv);
  }
}

}  // namespace b200kv

using namespace b200kv;

static int check_rows(const b200dec_rows* r) {
  if (!r) return B200KV_E_NULL;
  if (r->num_rows < 0) return B200KV_E_SHAPE;
  if ((r->seq_ids == nullptr) != (r->positions == nullptr)) return B200KV_E_NULL;
  if (!r->seq_ids && (!r->cached_lens || !r->num_decoding)) return B200KV_E_NULL;
  return B200KV_OK;
}

extern "C" int b200dec_rope_write(const void* qkv, int64_t qkv_stride, const b200dec_rows* rows, const b200dec_cache* cache,
                                  const b200kv_table* table, const float* cos_sin, int32_t table_len, int32_t half, int32_t heads,
                                  int32_t write_kv, int32_t unit_norm, float eps, void* q_out, int32_t* status, void* stream) {
  if (rows && rows->num_rows == 0) return B200KV_OK;
  if (!qkv || !q_out) return B200KV_E_NULL;
  int rc = check_rows(rows);
  if (rc == B200KV_OK) rc = check_dec_cache(cache, table);
  if (rc != B200KV_OK) return rc;
  if (half < 0 || 2 * half > cache->k_dim || (half > 0 && (!cos_sin || table_len < 1))) return B200KV_E_SHAPE;
  if (heads < 1 || heads % cache->kv_heads || cache->k_row > 64 * kRwMaxPairs || cache->v_row > 64 * kRwMaxPairs) return B200KV_E_SHAPE;
  if (!aligned(q_out, 16) || !aligned(cos_sin, 8)) return B200KV_E_ALIGN;
  const long long items = (long long)rows->num_rows * (heads + (write_kv ? 2 * cache->kv_heads : 0));
  const long long blocks = (items + kRwWarps - 1) / kRwWarps;
  if (items > 0x7FFFFFF0ll) return B200KV_E_RANGE;
  const DecCache c = dec_view(cache, table);
  cudaStream_t s = (cudaStream_t)stream;
  const bool pairs = cache->k_dim % 2 == 0 && cache->v_dim % 2 == 0 && half % 2 == 0 && qkv_stride % 2 == 0 &&
                     aligned(qkv, 2 * cache->elem) && aligned(cos_sin, 16);
  auto run = [&](auto* kernel, auto* in, auto* q) {
    return launch_result(launch_chained(kernel, dim3((unsigned)blocks), dim3(kRwWarps * 32), 0, s, in, (long long)qkv_stride, *rows, c, cos_sin,
                                        table_len, half, heads, write_kv, unit_norm, eps, q, status));
  };
  if (cache->elem == 2) {
    if (pairs && cache->k_row <= 128 && cache->v_row <= 128) return run(rope_write_kernel<uint16_t, true, 2>, (const uint16_t*)qkv, (uint16_t*)q_out);
    return run(pairs ? rope_write_kernel<uint16_t, true, kRwMaxPairs> : rope_write_kernel<uint16_t, false, kRwMaxPairs>, (const uint16_t*)qkv,
               (uint16_t*)q_out);
  }
  return run(pairs ? rope_write_kernel<float, true, kRwMaxPairs> : rope_write_kernel<float, false, kRwMaxPairs>, (const float*)qkv, (float*)q_out);
}

extern "C" int b200dec_norm_rope_write(const void* qkv, int64_t qkv_stride, const b200dec_rows* rows, const b200dec_cache* cache,
                                       const b200kv_table* table, const float* q_norm, const float* k_norm, float eps,
                                       const float* cos_sin, int32_t table_len, int32_t half, int32_t heads, void* q_out, int32_t* status,
                                       void* stream) {
  if (rows && rows->num_rows == 0) return B200KV_OK;
  if (!qkv || !q_out || !q_norm || !k_norm) return B200KV_E_NULL;
  int rc = check_rows(rows);
  if (rc == B200KV_OK) rc = check_dec_cache(cache, table);
  if (rc != B200KV_OK) return rc;
  if (half < 0 || 2 * half > cache->k_dim || (half > 0 && (!cos_sin || table_len < 1))) return B200KV_E_SHAPE;
  if (heads < 1 || heads % cache->kv_heads) return B200KV_E_SHAPE;
  if (!aligned(q_out, 16) || !aligned(cos_sin, 8)) return B200KV_E_ALIGN;
  const DecCache c = dec_view(cache, table);
  cudaStream_t s = (cudaStream_t)stream;
  const bool even = cache->k_dim % 2 == 0 && cache->v_dim % 2 == 0 && qkv_stride % 2 == 0 && aligned(qkv, 2 * cache->elem) &&
                    aligned(q_norm, 8) && aligned(k_norm, 8);
  const long long pairs = ((long long)(heads + cache->kv_heads) * cache->k_dim + (long long)cache->kv_heads * cache->v_dim) / 2;
  auto log2_of = [](int n) {
    for (int i = 0; i < 30; ++i)
      if (n == 1 << i) return i;
    return -1;
  };
  auto run = [&](auto* kernel, auto* in, auto* q) {
    return launch_result(launch_chained(kernel, dim3(rows->num_rows), dim3(kNrThreads), 0, s, in, (long long)qkv_stride, *rows, c, q_norm,
                                        k_norm, eps, cos_sin, table_len, half, heads, log2_of(cache->k_dim / 2), log2_of(cache->v_dim / 2), q,
                                        status));
  };
  const int keep = !even ? 0 : pairs <= 4 * kNrThreads ? 4 : pairs <= 8 * kNrThreads ? 8 : pairs <= 16 * kNrThreads ? 16 : 0;
  if (cache->elem == 2)
    return run(keep == 4   ? norm_rope_write_kernel<uint16_t, 4>
               : keep == 8 ? norm_rope_write_kernel<uint16_t, 8>
               : keep      ? norm_rope_write_kernel<uint16_t, 16> : norm_rope_write_kernel<uint16_t, 0>,
               (const uint16_t*)qkv, (uint16_t*)q_out);
  return run(keep == 4   ? norm_rope_write_kernel<float, 4>
             : keep == 8 ? norm_rope_write_kernel<float, 8>
             : keep      ? norm_rope_write_kernel<float, 16> : norm_rope_write_kernel<float, 0>,
             (const float*)qkv, (float*)q_out);
}

extern "C" int b200dec_attn_rows_opt(const void* q, const b200dec_cache* cache, const b200kv_table* table, const b200dec_rows* rows,
                                     int32_t heads, float scale, const b200dec_attn_options* options, void* out, int32_t* status,
                                     void* stream) {
  if (rows && rows->num_rows == 0) return B200KV_OK;
  if (!q || !out) return B200KV_E_NULL;
  int rc = check_rows(rows);
  if (rc == B200KV_OK) rc = check_dec_cache(cache, table);
  DecAttnOpt opt;
  if (rc == B200KV_OK) rc = dec_attn_opt(options, heads, cache->v_dim, &opt);
  if (rc != B200KV_OK) return rc;
  if (heads < 1 || heads % cache->kv_heads || cache->v_dim > kArThreads * kArPieces || cache->k_dim > 1024) return B200KV_E_SHAPE;
  if ((long long)cache->num_pages * cache->page_size > 0x7FFFFFFFll || rows->num_rows > 65535) return B200KV_E_RANGE;
  const size_t smem = (size_t)((cache->k_dim + 3) / 4 * 4 + 2 * kArKeys) * 4;
  const DecCache c = dec_view(cache, table);
  cudaStream_t s = (cudaStream_t)stream;
  if (cache->elem == 2)
    return launch_result(launch_chained(attn_rows_kernel<uint16_t>, dim3(heads, rows->num_rows), dim3(kArThreads), smem, s,
                                        (const uint16_t*)q, c, *rows, heads, scale, opt, (uint16_t*)out, status));
  return launch_result(launch_chained(attn_rows_kernel<float>, dim3(heads, rows->num_rows), dim3(kArThreads), smem, s, (const float*)q, c,
                                      *rows, heads, scale, opt, (float*)out, status));
}

extern "C" int b200dec_attn_rows(const void* q, const b200dec_cache* cache, const b200kv_table* table, const b200dec_rows* rows,
                                 int32_t heads, float scale, void* out, int32_t* status, void* stream) {
  return b200dec_attn_rows_opt(q, cache, table, rows, heads, scale, nullptr, out, status, stream);
}
