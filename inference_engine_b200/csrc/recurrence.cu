// Recurrent layers: a matrix state S [dim, vdim] per (request slot, head), kept in 32-bit, moved on by one token as
//   S <- decay * S;  u = beta (v - S^T k)  or  step * v;  S <- S + k u^T;  o = S^T q (+ skip v)
// behind a short causal convolution per channel with silu.  o comes from the decayed state before the write:
// o = (decay S)^T q + (k . q) u, so the two reductions over dim are made in one pass.
//   decode  one block per (entry, head): convolution, norms, decays, state and (optionally) the gated output norm in one
//           kernel.  HBM-bound: the state is read once and written once.
//   conv    prompt portions: silu(convolution) of every channel.
//   scan    prompt portions, token after token, the state in registers: any sizes, both precisions.
// The convolution's last inputs are kept by position modulo taps: a token writes the place that no token of its own
// convolution window reads, so a decode step needs no second buffer.
#include "recurrence.cuh"

namespace b200kv {

constexpr int kRdThreads = 256;

struct RecNorm {  // the output norm of the decode kernel
  const float* weight;  // [vdim]; NULL: raw fp32 output
  const void* gate;
  long long gate_stride, out_stride;
  float eps;
};

// Sum over the block; every thread gets it.
__device__ __forceinline__ float rd_sum(float v, float* part) {
  v = warp_sum(v);
  __syncthreads();
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kRdThreads / 32; ++i) t += part[i];
  return t;
}

// Threads are laid out as `rg` groups of rows by `cg` columns of four state entries; a thread owns rows r, r + rg, ...
// kRows > 0: its entries stay in registers between the reduction and the update; 0: any size, the state is read twice.
template <typename T, int kRows>
__global__ void __launch_bounds__(kRdThreads)
recurrence_decode_kernel(const b200dec_recurrence rec, const b200dec_recurrence_in in, const b200dec_entries ent, const RecNorm norm,
                         void* __restrict__ out, int cg, int rg, int32_t* status) {
  extern __shared__ __align__(16) float rd_smem[];
  pdl_enter();
  const int h = blockIdx.x, e = blockIdx.y, tid = threadIdx.x;
  const int D = rec.dim, P = rec.vdim, P4 = rec_round4(P), Dp = rec_round4(D);
  float* qs = rd_smem;                 // [Dp]
  float* ks = qs + Dp;                 // [Dp]
  float* gs = ks + Dp;                 // [Dp] decay of each row
  float* vs = gs + Dp;                 // [P4]
  float* us = vs + P4;                 // [P4]
  float* os = us + P4;                 // [P4]
  float* red = os + P4;                // [2][rg][4 * cg]
  __shared__ float part[kRdThreads / 32];
  const int nd = min(*ent.num_decoding, ent.num_entries);
  if (e >= nd) {  // idle; in a pure decode step the row is cleared
    pdl_wait();
    if (!ent.cu_seqlens && e < ent.num_rows)
      for (int p = tid; p < P; p += kRdThreads) {
        if (norm.weight) st_elem((T*)out + e * norm.out_stride + h * P + p, 0.f);
        else ((float*)out)[((long long)e * rec.heads + h) * P + p] = 0.f;
      }
    return;
  }
  const RecEntry x = rec_entry(ent, rec, e, status);
  pdl_wait();
  if (x.n == 0) return;
  const int c4 = tid % cg, r0 = tid / cg;
  const bool mine = r0 < rg;
  float* state = rec.state + ((long long)x.slot * rec.heads + h) * D * P4;
  float4 S[kRows > 0 ? kRows : 1];
  if (kRows > 0) {
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int d = r0 + i * rg;
      S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (mine && d < D && x.pos > 0) S[i] = __ldcg(reinterpret_cast<const float4*>(state + (long long)d * P4) + c4);
    }
  }
  // ---- the token's q, k, v (convolution and silu), decays and step
  const int per = rec.heads / rec.qk_heads, hq = h / per;
  const T* xr = (const T*)in.x + x.first * in.x_stride;
  T* ring = (T*)rec.ring + (long long)x.slot * rec.taps * rec.channels;
  const int now = x.pos % rec.taps;
  const bool first_of_group = h % per == 0;
  auto conv = [&](int ch, bool keep) {
    const T raw = xr[ch];
    if (keep) ring[(long long)now * rec.channels + ch] = raw;
    return rec_conv(rec, ch, x.pos, ld_elem(&raw), [&](int j) {
      int at = now - j;
      if (at < 0) at += rec.taps;
      return ldcg_elem(ring + (long long)at * rec.channels + ch);
    });
  };
  const float na = rec.neg_a[h];
  float step = 0.f;
  if (!rec.channel_decay) step = softplus_f(ld_elem((const T*)in.step + x.first * in.step_stride + h) + rec.dt_bias[h]);
  const float decay_all = expf(na * step);
  float sq = 0.f, sk = 0.f, qk = 0.f;
  for (int i = tid; i < 2 * Dp + P4; i += kRdThreads) {
    if (i < 2 * Dp) {
      const bool is_q = i < Dp;
      const int d = is_q ? i : i - Dp;
      float v = 0.f;
      if (d < D) v = conv((is_q ? rec.off_q : rec.off_k) + hq * D + d, first_of_group);
      (is_q ? qs : ks)[d] = v;
      if (is_q) sq = fmaf(v, v, sq);
      else {
        sk = fmaf(v, v, sk);
        float g = decay_all;
        if (rec.channel_decay && d < D)
          g = expf(na * softplus_f(ld_elem((const T*)in.step + x.first * in.step_stride + h * D + d) + rec.dt_bias[h * D + d]));
        gs[d] = g;
      }
    } else {
      const int p = i - 2 * Dp;
      vs[p] = p < P ? conv(rec.off_v + h * P + p, true) : 0.f;
    }
  }
  if (rec.unit_norm) {
    sq = rd_sum(sq, part);
    sk = rd_sum(sk, part);
  } else {
    __syncthreads();
  }
  const float fq = rec.q_scale * (rec.unit_norm ? 1.0f / sqrtf(sq + rec.unit_eps) : 1.f);
  const float fk = rec.unit_norm ? 1.0f / sqrtf(sk + rec.unit_eps) : 1.f;
  for (int d = tid; d < D; d += kRdThreads) {
    qs[d] *= fq;
    ks[d] *= fk;
    qk = fmaf(qs[d], ks[d], qk);
  }
  qk = rd_sum(qk, part);
  const float beta = rec.correct ? sigmoid_f(ld_elem((const T*)in.beta + x.first * in.beta_stride + h)) : step;
  const float skip = rec.skip ? rec.skip[h] : 0.f;
  // ---- (decay S)^T k and (decay S)^T q, then the update, in slabs of 4 * cg columns
  float ss = 0.f;
  for (int col0 = 0; col0 < P4; col0 += 4 * cg) {
    const int col = col0 + 4 * c4;
    const bool in_row = mine && col < P4;
    float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
    auto add = [&](float4& s, int d) {
      const float g = gs[d], k = ks[d], q = qs[d];
      s.x *= g; s.y *= g; s.z *= g; s.w *= g;
      ak.x = fmaf(s.x, k, ak.x); ak.y = fmaf(s.y, k, ak.y); ak.z = fmaf(s.z, k, ak.z); ak.w = fmaf(s.w, k, ak.w);
      aq.x = fmaf(s.x, q, aq.x); aq.y = fmaf(s.y, q, aq.y); aq.z = fmaf(s.z, q, aq.z); aq.w = fmaf(s.w, q, aq.w);
    };
    if (in_row) {
      if (kRows > 0) {
#pragma unroll
        for (int i = 0; i < kRows; ++i)
          if (r0 + i * rg < D) add(S[i], r0 + i * rg);
      } else if (x.pos > 0) {
        for (int d = r0; d < D; d += rg) {
          float4 s = __ldcg(reinterpret_cast<const float4*>(state + (long long)d * P4 + col));
          add(s, d);
        }
      }
      *reinterpret_cast<float4*>(red + r0 * 4 * cg + 4 * c4) = ak;
      *reinterpret_cast<float4*>(red + (rg + r0) * 4 * cg + 4 * c4) = aq;
    }
    __syncthreads();
    for (int i = tid; i < 4 * cg && col0 + i < P4; i += kRdThreads) {
      float rk = 0.f, rq = 0.f;
      for (int r = 0; r < rg; ++r) {
        rk += red[r * 4 * cg + i];
        rq += red[(rg + r) * 4 * cg + i];
      }
      const float v = vs[col0 + i];
      const float u = rec.correct ? beta * (v - rk) : beta * v;
      us[col0 + i] = u;
      const float o = fmaf(skip, v, fmaf(qk, u, rq));
      os[col0 + i] = o;
      ss = fmaf(o, o, ss);
    }
    __syncthreads();
    if (in_row) {
      const float4 u = *reinterpret_cast<const float4*>(us + col);
      auto move = [&](float4 s, int d) {
        const float k = ks[d];
        s.x = fmaf(k, u.x, s.x); s.y = fmaf(k, u.y, s.y); s.z = fmaf(k, u.z, s.z); s.w = fmaf(k, u.w, s.w);
        *reinterpret_cast<float4*>(state + (long long)d * P4 + col) = s;
      };
      if (kRows > 0) {
#pragma unroll
        for (int i = 0; i < kRows; ++i)
          if (r0 + i * rg < D) move(S[i], r0 + i * rg);
      } else {
        for (int d = r0; d < D; d += rg) {
          float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
          if (x.pos > 0) s = __ldcg(reinterpret_cast<const float4*>(state + (long long)d * P4 + col));
          const float g = gs[d];
          s.x *= g; s.y *= g; s.z *= g; s.w *= g;
          move(s, d);
        }
      }
    }
  }
  // ---- output
  if (!norm.weight) {
    for (int p = tid; p < P; p += kRdThreads) ((float*)out)[((long long)x.first * rec.heads + h) * P + p] = os[p];
    return;
  }
  const float inv = 1.0f / sqrtf(rd_sum(ss, part) / (float)P + norm.eps);
  const T* gate = (const T*)norm.gate + x.first * norm.gate_stride + h * P;
  T* dst = (T*)out + x.first * norm.out_stride + h * P;
  for (int p = tid; p < P; p += kRdThreads) st_elem(dst + p, os[p] * inv * norm.weight[p] * sigmoid_f(ld_elem(gate + p)));
}

// ---------------------------------------------------------------- convolution of prompt portions
constexpr int kRcThreads = 256;

// kVec channels (8, or 1 for any size) of one row per thread.
template <typename T, int kVec>
__global__ void __launch_bounds__(kRcThreads)
conv_rows_kernel(const b200dec_recurrence rec, const b200dec_recurrence_in in, const b200dec_entries ent, T* __restrict__ out,
                 int out_stride, int32_t* status) {
  pdl_enter();
  const int r = blockIdx.y, ch = (blockIdx.x * kRcThreads + threadIdx.x) * kVec;
  const int e = ent.seq_ids[r];
  if (e < *ent.num_decoding || e >= ent.num_entries || ch >= rec.channels) return;
  const int pos = ent.positions[r], first = ent.cu_seqlens[e], slot = ent.slots[e];
  if (slot < 0 || slot >= rec.num_slots || pos < 0 || first < 0 || first > r) {
    if (slot != -1 && threadIdx.x == 0 && status) atomicOr(status, B200KV_S_BAD_POSITION);
    return;
  }
  pdl_wait();
  const T* ring = (const T*)rec.ring + (long long)slot * rec.taps * rec.channels + ch;
  float acc[kVec], f[kVec];
  auto load = [&](const T* p, bool fresh) {
    if constexpr (kVec == 1) {
      f[0] = fresh ? ldcg_elem(p) : ld_elem(p);
    } else {
#pragma unroll
      for (int i = 0; i < kVec; i += 4) {
        float t[4];
        if constexpr (sizeof(T) == 2) {
          const uint2 v = fresh ? __ldcg(reinterpret_cast<const uint2*>(p + i)) : *reinterpret_cast<const uint2*>(p + i);
          t[0] = __uint_as_float(v.x << 16); t[1] = __uint_as_float(v.x & 0xFFFF0000u);
          t[2] = __uint_as_float(v.y << 16); t[3] = __uint_as_float(v.y & 0xFFFF0000u);
        } else {
          ld_fresh4(p + i, t);
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) f[i + k] = t[k];
      }
    }
  };
#pragma unroll
  for (int i = 0; i < kVec; ++i) acc[i] = rec.conv_b ? rec.conv_b[ch + i] : 0.f;
  const int back = min(rec.taps - 1, pos);
  for (int j = 0; j <= back; ++j) {
    if (r - j >= first) load((const T*)in.x + (long long)(r - j) * in.x_stride + ch, false);
    else load(ring + (long long)((pos - j) % rec.taps) * rec.channels, true);
    const float* w = rec.conv_w + (long long)(rec.taps - 1 - j) * rec.channels + ch;
#pragma unroll
    for (int i = 0; i < kVec; ++i) acc[i] = fmaf(w[i], f[i], acc[i]);
  }
  T* dst = out + (long long)r * out_stride + ch;
#pragma unroll
  for (int i = 0; i < kVec; ++i) acc[i] = silu_f(acc[i]);
  if constexpr (kVec == 1) {
    st_elem(dst, acc[0]);
  } else {
#pragma unroll
    for (int i = 0; i < kVec; i += 4) {
      const float t[4] = {acc[i], acc[i + 1], acc[i + 2], acc[i + 3]};
      st_elem4(dst + i, t);
    }
  }
}

// The raw inputs of the last `taps` positions of an entry's portion go into its ring; block `part` of `parts` does its share.
template <typename T>
__device__ __forceinline__ void rec_keep_inputs(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const RecEntry& x, int part,
                                                int parts, int threads) {
  const int keep = min(rec.taps, x.n);
  T* ring = (T*)rec.ring + (long long)x.slot * rec.taps * rec.channels;
  for (int j = 0; j < keep; ++j) {
    const int row = x.first + x.n - 1 - j, at = (x.pos + x.n - 1 - j) % rec.taps;
    for (int c = part * threads + threadIdx.x; c < rec.channels; c += parts * threads)
      ring[(long long)at * rec.channels + c] = ((const T*)in.x)[row * in.x_stride + c];
  }
}

// ---------------------------------------------------------------- scan of prompt portions, token after token
constexpr int kRsThreads = 256;
constexpr int kRsTokens = 16;  // tokens prepared in shared memory at a time

// kLanes lanes share a state column; a lane owns rows 4 * lane + 4 * kLanes * j + (0..3).  One block: kRsThreads / kLanes
// columns of one head of one entry.
template <typename T, int kRows, int kLanes>
__global__ void __launch_bounds__(kRsThreads)
recurrence_scan_kernel(const b200dec_recurrence rec, const b200dec_recurrence_in in, const T* __restrict__ conv, int conv_stride,
                       const b200dec_entries ent, float* __restrict__ out, int slabs, int32_t* status) {
  constexpr int kDim = kRows * kLanes, kCols = kRsThreads / kLanes;
  extern __shared__ __align__(16) float rs_smem[];
  float* qs = rs_smem;                      // [kRsTokens][kDim]
  float* ks = qs + kRsTokens * kDim;
  float* gs = ks + kRsTokens * kDim;
  float* vs = gs + kRsTokens * kDim;        // [kRsTokens][kCols]
  float* cf = vs + kRsTokens * kCols;       // [kRsTokens] beta or step
  float* kq = cf + kRsTokens;               // [kRsTokens] k . q
  pdl_enter();
  const int e = blockIdx.y, h = blockIdx.x / slabs, slab = blockIdx.x - h * slabs, tid = threadIdx.x;
  const int warp = tid >> 5, wl = tid & 31;
  if (e < *ent.num_decoding) { pdl_wait(); return; }
  const RecEntry x = rec_entry(ent, rec, e, status);
  pdl_wait();
  if (x.n == 0) return;
  const int D = rec.dim, P = rec.vdim, P4 = rec_round4(P), hq = h / (rec.heads / rec.qk_heads);
  const int lane = tid % kLanes, col = tid / kLanes, p = slab * kCols + col;
  float* state = rec.state + ((long long)x.slot * rec.heads + h) * D * P4;
  float S[kRows];
#pragma unroll
  for (int i = 0; i < kRows; ++i) {
    const int d = (i / 4) * 4 * kLanes + 4 * lane + (i & 3);
    S[i] = x.pos > 0 && d < D && p < P ? __ldcg(state + (long long)d * P4 + p) : 0.f;
  }
  const float na = rec.neg_a[h], skip = rec.skip ? rec.skip[h] : 0.f;
  const float b_all = rec.channel_decay ? 0.f : rec.dt_bias[h];
  for (int t0 = 0; t0 < x.n; t0 += kRsTokens) {
    const int nt = min(kRsTokens, x.n - t0);
    __syncthreads();
    for (int t = warp; t < nt; t += kRsThreads / 32) {
      const long long row = x.first + t0 + t;
      const T* src = conv + row * conv_stride;
      float sq = 0.f, sk = 0.f, dot = 0.f;
      float step = 0.f;
      if (!rec.channel_decay) step = softplus_f(ld_elem((const T*)in.step + row * in.step_stride + h) + b_all);
      const float decay_all = expf(na * step);
      for (int d = wl; d < kDim; d += 32) {
        float q = 0.f, k = 0.f, g = decay_all;
        if (d < D) {
          q = ld_elem(src + rec.off_q + hq * D + d);
          k = ld_elem(src + rec.off_k + hq * D + d);
          if (rec.channel_decay)
            g = expf(na * softplus_f(ld_elem((const T*)in.step + row * in.step_stride + h * D + d) + rec.dt_bias[h * D + d]));
        }
        qs[t * kDim + d] = q;
        ks[t * kDim + d] = k;
        gs[t * kDim + d] = g;
        sq = fmaf(q, q, sq);
        sk = fmaf(k, k, sk);
        dot = fmaf(q, k, dot);
      }
      sq = warp_sum(sq);
      sk = warp_sum(sk);
      dot = warp_sum(dot);
      const float fq = rec.q_scale * (rec.unit_norm ? 1.0f / sqrtf(sq + rec.unit_eps) : 1.f);
      const float fk = rec.unit_norm ? 1.0f / sqrtf(sk + rec.unit_eps) : 1.f;
      for (int d = wl; d < kDim; d += 32) {
        qs[t * kDim + d] *= fq;
        ks[t * kDim + d] *= fk;
      }
      for (int c = wl; c < kCols; c += 32)
        vs[t * kCols + c] = slab * kCols + c < P ? ld_elem(src + rec.off_v + h * P + slab * kCols + c) : 0.f;
      if (wl == 0) {
        kq[t] = dot * fq * fk;
        cf[t] = rec.correct ? sigmoid_f(ld_elem((const T*)in.beta + row * in.beta_stride + h)) : step;
      }
    }
    __syncthreads();
#pragma unroll 2
    for (int t = 0; t < nt; ++t) {
      float k[kRows], rk[4] = {0.f, 0.f, 0.f, 0.f}, rq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int j = 0; j < kRows / 4; ++j) {
        const int d = t * kDim + j * 4 * kLanes + 4 * lane;
        const float4 kk = *reinterpret_cast<const float4*>(ks + d), qq = *reinterpret_cast<const float4*>(qs + d);
        const float4 gg = *reinterpret_cast<const float4*>(gs + d);
        const float q[4] = {qq.x, qq.y, qq.z, qq.w}, g[4] = {gg.x, gg.y, gg.z, gg.w};
        k[4 * j] = kk.x; k[4 * j + 1] = kk.y; k[4 * j + 2] = kk.z; k[4 * j + 3] = kk.w;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          S[4 * j + i] *= g[i];
          rk[i] = fmaf(S[4 * j + i], k[4 * j + i], rk[i]);
          rq[i] = fmaf(S[4 * j + i], q[i], rq[i]);
        }
      }
      float sk = (rk[0] + rk[1]) + (rk[2] + rk[3]), sq = (rq[0] + rq[1]) + (rq[2] + rq[3]);
#pragma unroll
      for (int o = kLanes / 2; o > 0; o >>= 1) {
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
      }
      const float v = vs[t * kCols + col];
      const float u = rec.correct ? cf[t] * (v - sk) : cf[t] * v;
#pragma unroll
      for (int i = 0; i < kRows; ++i) S[i] = fmaf(k[i], u, S[i]);
      if (lane == 0 && p < P) out[((long long)(x.first + t0 + t) * rec.heads + h) * P + p] = fmaf(skip, v, fmaf(kq[t], u, sq));
    }
  }
#pragma unroll
  for (int i = 0; i < kRows; ++i) {
    const int d = (i / 4) * 4 * kLanes + 4 * lane + (i & 3);
    if (d < D && p < P4) state[(long long)d * P4 + p] = p < P ? S[i] : 0.f;
  }
  rec_keep_inputs<T>(rec, in, x, blockIdx.x, gridDim.x, kRsThreads);
}

template <typename T, int kRows>
static int rd_launch(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const b200dec_entries& ent, const RecNorm& norm, void* out,
                     int cg, int rg, int32_t* status, cudaStream_t s) {
  const size_t smem = (size_t)(3 * rec_round4(rec.dim) + 3 * rec_round4(rec.vdim) + 8 * rg * cg) * 4;
  if (smem > 200 * 1024) return B200KV_E_RANGE;
  if (cudaFuncSetAttribute(recurrence_decode_kernel<T, kRows>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return B200KV_E_LAUNCH;
  return launch_result(launch_chained(recurrence_decode_kernel<T, kRows>, dim3(rec.heads, ent.num_entries), dim3(kRdThreads), smem, s, rec, in,
                                      ent, norm, out, cg, rg, status));
}

template <typename T>
static int rd_run(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const b200dec_entries& ent, const RecNorm& norm, void* out,
                  int32_t* status, cudaStream_t s) {
  const int quads = rec_round4(rec.vdim) / 4, cg = quads < kRdThreads ? quads : kRdThreads, rg = kRdThreads / cg;
  const int rows = (rec.dim + rg - 1) / rg;
  if (quads <= kRdThreads && rows <= 4) return rd_launch<T, 4>(rec, in, ent, norm, out, cg, rg, status, s);
  if (quads <= kRdThreads && rows <= 8) return rd_launch<T, 8>(rec, in, ent, norm, out, cg, rg, status, s);
  if (quads <= kRdThreads && rows <= 16) return rd_launch<T, 16>(rec, in, ent, norm, out, cg, rg, status, s);
  return rd_launch<T, 0>(rec, in, ent, norm, out, cg, rg, status, s);
}

template <typename T, int kRows, int kLanes>
static int rs_launch(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const void* conv, const b200dec_entries& ent, float* out,
                     int32_t* status, cudaStream_t s) {
  constexpr int kCols = kRsThreads / kLanes;
  const int slabs = (rec.vdim + kCols - 1) / kCols;
  const size_t smem = (size_t)(kRsTokens * (3 * kRows * kLanes + kCols + 2)) * 4;
  if (smem > 200 * 1024) return B200KV_E_RANGE;
  if (cudaFuncSetAttribute(recurrence_scan_kernel<T, kRows, kLanes>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return B200KV_E_LAUNCH;
  return launch_result(launch_chained(recurrence_scan_kernel<T, kRows, kLanes>, dim3(rec.heads * slabs, ent.num_entries), dim3(kRsThreads), smem,
                                      s, rec, in, (const T*)conv, (rec.channels + 7) / 8 * 8, ent, out, slabs, status));
}

template <typename T>
static int rs_run(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const void* conv, const b200dec_entries& ent, float* out,
                  int32_t* status, cudaStream_t s) {
  const int D = rec.dim;
  if (D <= 32) return rs_launch<T, 4, 8>(rec, in, conv, ent, out, status, s);
  if (D <= 64) return rs_launch<T, 8, 8>(rec, in, conv, ent, out, status, s);
  if (D <= 128) return rs_launch<T, 16, 8>(rec, in, conv, ent, out, status, s);
  if (D <= 256) return rs_launch<T, 16, 16>(rec, in, conv, ent, out, status, s);
  if (D <= 512) return rs_launch<T, 16, 32>(rec, in, conv, ent, out, status, s);
  if (D <= 1024) return rs_launch<T, 32, 32>(rec, in, conv, ent, out, status, s);
  return B200KV_E_SHAPE;
}

template <typename T>
static int rc_run(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const b200dec_entries& ent, void* out, int32_t* status,
                  cudaStream_t s) {
  const bool vec = rec.channels % 8 == 0 && in.x_stride % 8 == 0 && aligned(in.x, 16) && aligned(rec.ring, 16) && aligned(out, 16);
  const int items = vec ? rec.channels / 8 : rec.channels;
  auto* kernel = vec ? conv_rows_kernel<T, 8> : conv_rows_kernel<T, 1>;
  return launch_result(launch_chained(kernel, dim3((items + kRcThreads - 1) / kRcThreads, ent.num_rows), dim3(kRcThreads), 0, s, rec, in, ent,
                                      (T*)out, (rec.channels + 7) / 8 * 8, status));
}

}  // namespace b200kv

using namespace b200kv;

extern "C" int b200dec_recurrence_decode(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const b200dec_entries* ent,
                                         const float* norm_w, float eps, const void* gate, int64_t gate_stride, void* out,
                                         int64_t out_stride, int32_t* status, void* stream) {
  const int rc = check_recurrence(rec, in, ent);
  if (rc != B200KV_OK) return rc;
  if (ent->num_entries == 0) return B200KV_OK;
  if (!out || (norm_w && !gate)) return B200KV_E_NULL;
  const RecNorm norm{norm_w, gate, gate_stride, out_stride, eps};
  cudaStream_t s = (cudaStream_t)stream;
  return rec->elem == 2 ? rd_run<uint16_t>(*rec, *in, *ent, norm, out, status, s) : rd_run<float>(*rec, *in, *ent, norm, out, status, s);
}

extern "C" int b200dec_conv_rows(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const b200dec_entries* ent, void* conv_out,
                                 int32_t* status, void* stream) {
  const int rc = check_recurrence(rec, in, ent);
  if (rc != B200KV_OK) return rc;
  if (!ent->cu_seqlens || !conv_out) return B200KV_E_NULL;
  if (ent->num_rows == 0) return B200KV_OK;
  if (ent->num_rows > 65535) return B200KV_E_RANGE;
  cudaStream_t s = (cudaStream_t)stream;
  return rec->elem == 2 ? rc_run<uint16_t>(*rec, *in, *ent, conv_out, status, s) : rc_run<float>(*rec, *in, *ent, conv_out, status, s);
}

extern "C" int b200dec_recurrence_scan(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const void* conv_out,
                                       const b200dec_entries* ent, float* out, int32_t* status, void* stream) {
  const int rc = check_recurrence(rec, in, ent);
  if (rc != B200KV_OK) return rc;
  if (!ent->cu_seqlens || !conv_out || !out) return B200KV_E_NULL;
  if (ent->num_entries == 0 || ent->num_rows == 0) return B200KV_OK;
  cudaStream_t s = (cudaStream_t)stream;
  return rec->elem == 2 ? rs_run<uint16_t>(*rec, *in, conv_out, *ent, out, status, s)
                        : rs_run<float>(*rec, *in, conv_out, *ent, out, status, s);
}
