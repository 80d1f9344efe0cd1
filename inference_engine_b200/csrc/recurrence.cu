// Recurrent layers: a matrix state S [dim, vdim] per (request slot, head), kept in 32-bit, moved on by one token as
//   S <- decay * S;  u = beta (v - S^T k)  or  step * v;  S <- S + k u^T;  o = S^T q (+ skip v)
// behind a short causal convolution per channel with silu.  o comes from the decayed state before the write:
// o = (decay S)^T q + (k . q) u, so the two reductions over dim are made in one pass.
//   decode  one block per (entry, head): convolution, norms, decays, state and (optionally) the gated output norm in one
//           kernel, for states of any size (recurrence_decode.cu has the one for the usual sizes).
//   conv    prompt portions: silu(convolution) of every channel.
//   scan    prompt portions, token after token, the state in registers: any sizes, both precisions.
// The convolution's last inputs are kept by position modulo taps: a token writes the place that no token of its own
// convolution window reads, so a decode step needs no second buffer.
#include "recurrence.cuh"

namespace b200kv {

constexpr int kRdThreads = 256;

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
// The state is read twice, for the reduction and for the update, so that it may have any size.
template <typename T>
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
  __shared__ float part[3 * kRdThreads / 32];
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
  // ---- the token's q, k, v (convolution and silu), decays and step; two channels per thread at a time, all loads of
  // both ahead of the arithmetic
  const int per = rec.heads / rec.qk_heads, hq = h / per;
  const T* xr = (const T*)in.x + x.first * in.x_stride;
  const T* sr = (const T*)in.step + x.first * in.step_stride;
  T* ring = (T*)rec.ring + (long long)x.slot * rec.taps * rec.channels;
  const int now = x.pos % rec.taps, back = min(rec.taps - 1, x.pos);
  const bool first_of_group = h % per == 0;
  const float na = rec.neg_a[h];
  float step = 0.f;
  if (!rec.channel_decay) step = ld_elem(sr + h) + rec.dt_bias[h];
  const float beta_in = rec.correct ? ld_elem((const T*)in.beta + x.first * in.beta_stride + h) : 0.f;
  float sq = 0.f, sk = 0.f, qk = 0.f;
  const int total = 2 * Dp + P4;
  constexpr int kNear = 4;  // taps handled without a loop
  for (int base = tid; base < total; base += 2 * kRdThreads) {
    float xv[2][kNear], wv[2][kNear], bv[2], dv[2];
    int ch[2];
    T raw[2];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = base + u * kRdThreads, d = i < Dp ? i : i - Dp;
      ch[u] = -1;
      if (i < Dp) { if (d < D) ch[u] = rec.off_q + hq * D + d; }
      else if (i < 2 * Dp) { if (d < D) ch[u] = rec.off_k + hq * D + d; }
      else if (i < total && i - 2 * Dp < P) ch[u] = rec.off_v + h * P + i - 2 * Dp;
      if (ch[u] < 0) continue;
      raw[u] = xr[ch[u]];
      bv[u] = rec.conv_b ? rec.conv_b[ch[u]] : 0.f;
      dv[u] = 0.f;
      if (rec.channel_decay && i >= Dp && i < 2 * Dp) dv[u] = ld_elem(sr + h * D + d) + rec.dt_bias[h * D + d];
#pragma unroll
      for (int j = 0; j < kNear; ++j) {
        xv[u][j] = wv[u][j] = 0.f;
        if (j > back) continue;
        int at = now - j;
        if (at < 0) at += rec.taps;
        wv[u][j] = rec.conv_w[(long long)(rec.taps - 1 - j) * rec.channels + ch[u]];
        if (j > 0) xv[u][j] = ldcg_elem(ring + (long long)at * rec.channels + ch[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int i = base + u * kRdThreads;
      if (i >= total) break;
      float v = 0.f;
      if (ch[u] >= 0) {
        xv[u][0] = ld_elem(&raw[u]);
        v = bv[u];
#pragma unroll
        for (int j = 0; j < kNear; ++j) v = fmaf(wv[u][j], xv[u][j], v);
        for (int j = kNear; j <= back; ++j) {
          int at = now - j;
          if (at < 0) at += rec.taps;
          v = fmaf(rec.conv_w[(long long)(rec.taps - 1 - j) * rec.channels + ch[u]], ldcg_elem(ring + (long long)at * rec.channels + ch[u]), v);
        }
        v *= sigmoid_act<T>(v);
        if (i >= 2 * Dp || first_of_group) ring[(long long)now * rec.channels + ch[u]] = raw[u];
      }
      if (i < Dp) {
        qs[i] = v;
        sq = fmaf(v, v, sq);
      } else if (i < 2 * Dp) {
        ks[i - Dp] = v;
        sk = fmaf(v, v, sk);
        if (rec.channel_decay) gs[i - Dp] = ch[u] >= 0 ? expf(na * softplus_f(dv[u])) : 1.f;
      } else {
        vs[i - 2 * Dp] = v;
      }
    }
  }
  if (!rec.channel_decay) {
    step = softplus_f(step);
    const float g = expf(na * step);
    for (int d = tid; d < Dp; d += kRdThreads) gs[d] = g;
  }
  __syncthreads();
  for (int d = tid; d < D; d += kRdThreads) qk = fmaf(qs[d], ks[d], qk);
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  qk = warp_sum(qk);
  if ((tid & 31) == 0) {
    part[tid >> 5] = sq;
    part[8 + (tid >> 5)] = sk;
    part[16 + (tid >> 5)] = qk;
  }
  __syncthreads();
  sq = sk = qk = 0.f;
#pragma unroll
  for (int i = 0; i < kRdThreads / 32; ++i) {
    sq += part[i];
    sk += part[8 + i];
    qk += part[16 + i];
  }
  // the factors of q and k are applied to the sums, not to the vectors
  const float fq = rec.q_scale * (rec.unit_norm ? 1.0f / sqrtf(sq + rec.unit_eps) : 1.f);
  const float fk = rec.unit_norm ? 1.0f / sqrtf(sk + rec.unit_eps) : 1.f;
  qk *= fq * fk;
  const float beta = rec.correct ? sigmoid_f(beta_in) : step;
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
      if (x.pos > 0) {
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
#pragma unroll 8
      for (int r = 0; r < rg; ++r) {
        rk += red[r * 4 * cg + i];
        rq += red[(rg + r) * 4 * cg + i];
      }
      const float v = vs[col0 + i];
      const float u = rec.correct ? beta * fmaf(-fk, rk, v) : beta * v;
      us[col0 + i] = fk * u;
      const float o = fmaf(skip, v, fmaf(qk, u, fq * rq));
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
      for (int d = r0; d < D; d += rg) {
        float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
        if (x.pos > 0) s = __ldcg(reinterpret_cast<const float4*>(state + (long long)d * P4 + col));
        const float g = gs[d];
        s.x *= g; s.y *= g; s.z *= g; s.w *= g;
        move(s, d);
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
constexpr int kRcThreads = 128;
constexpr int kRcRun = 8;  // rows per thread

// kVec channels (8, or 1 for any size) of kRcRun consecutive rows per thread.  kTaps > 0: the taps' weights and the rows'
// inputs are held in registers, so that every input is loaded once.  kTaps = 0: any number of taps, row by row.
template <typename T, int kVec, int kTaps>
__global__ void __launch_bounds__(kRcThreads)
conv_rows_kernel(const b200dec_recurrence rec, const b200dec_recurrence_in in, const b200dec_entries ent, T* __restrict__ out,
                 int out_stride, int32_t* status) {
  pdl_enter();
  const int r0 = blockIdx.x * kRcRun, ch = (blockIdx.y * kRcThreads + threadIdx.x) * kVec;
  if (ch >= rec.channels) return;
  const int nd = *ent.num_decoding;
  constexpr int kHold = kTaps > 0 ? kTaps : 1;
  float w[kHold][kVec], bias[kVec];
#pragma unroll
  for (int i = 0; i < kVec; ++i) bias[i] = rec.conv_b ? rec.conv_b[ch + i] : 0.f;
  if (kTaps > 0)
#pragma unroll
    for (int j = 0; j < kHold; ++j) ld_vec(rec.conv_w + (long long)j * rec.channels + ch, w[j]);
  pdl_wait();
  // Input j positions before row r (of an entry whose rows start at `first`), zero in front of the sequence.
  auto before = [&](int r, int j, int first, int pos, int slot, float (&f)[kVec]) {
    if (j > pos) {
#pragma unroll
      for (int i = 0; i < kVec; ++i) f[i] = 0.f;
    } else if (r - j >= first) {
      ld_vec((const T*)in.x + (long long)(r - j) * in.x_stride + ch, f);
    } else {
      const T* p = (const T*)rec.ring + ((long long)slot * rec.taps + (pos - j) % rec.taps) * rec.channels + ch;
      if constexpr (kVec == 1) {
        f[0] = ldcg_elem(p);
      } else if constexpr (sizeof(T) == 2) {
        unpack8(__ldcg(reinterpret_cast<const uint4*>(p)), f);
      } else {
        float a[4], b[4];
        ld_fresh4(p, a);
        ld_fresh4(p + 4, b);
#pragma unroll
        for (int i = 0; i < 4; ++i) { f[i] = a[i]; f[4 + i] = b[i]; }
      }
    }
  };
  auto put = [&](int r, float (&acc)[kVec]) {
#pragma unroll
    for (int i = 0; i < kVec; ++i) acc[i] *= sigmoid_act<T>(acc[i]);
    st_vec(out + (long long)r * out_stride + ch, acc);
  };
  const int rows = min(kRcRun, ent.num_rows - r0);
  float x[kRcRun + kHold - 1][kVec];  // inputs of rows r0 - (taps - 1) .. r0 + kRcRun - 1, as the entry at hand sees them
  if (kTaps > 0) {
#pragma unroll
    for (int t = 0; t < kRcRun; ++t)
      if (t < rows) ld_vec((const T*)in.x + (long long)(r0 + t) * in.x_stride + ch, x[t + kHold - 1]);
  }
  int e_last = -1;
#pragma unroll
  for (int t = 0; t < kRcRun; ++t) {
    if (t >= rows) break;
    const int r = r0 + t, e = ent.seq_ids[r];
    const bool fresh = e != e_last;
    e_last = e;
    if (e < nd || e >= ent.num_entries) continue;
    const int pos = ent.positions[r], first = ent.cu_seqlens[e], slot = ent.slots[e];
    if (slot < 0 || slot >= rec.num_slots || pos < 0 || first < 0 || first > r) {
      if (slot != -1 && ch == 0 && status) atomicOr(status, B200KV_S_BAD_POSITION);
      continue;
    }
    float acc[kVec];
#pragma unroll
    for (int i = 0; i < kVec; ++i) acc[i] = bias[i];
    if (kTaps > 0) {
      float h[kHold][kVec];
      if (fresh) {  // the first row of the thread or of an entry: its history comes from elsewhere
#pragma unroll
        for (int j = 1; j < kHold; ++j) before(r, j, first, pos, slot, h[j]);
      }
#pragma unroll
      for (int j = 1; j < kHold; ++j)
#pragma unroll
        for (int i = 0; i < kVec; ++i) {
          if (fresh) x[t + kHold - 1 - j][i] = h[j][i];
          acc[i] = fmaf(w[kHold - 1 - j][i], x[t + kHold - 1 - j][i], acc[i]);
        }
#pragma unroll
      for (int i = 0; i < kVec; ++i) acc[i] = fmaf(w[kHold - 1][i], x[t + kHold - 1][i], acc[i]);
    } else {
      for (int j = 0; j < rec.taps; ++j) {
        float f[kVec];
        before(r, j, first, pos, slot, f);
#pragma unroll
        for (int i = 0; i < kVec; ++i) acc[i] = fmaf(rec.conv_w[(long long)(rec.taps - 1 - j) * rec.channels + ch + i], f[i], acc[i]);
      }
    }
    put(r, acc);
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

template <typename T>
static int rd_run(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const b200dec_entries& ent, const RecNorm& norm, void* out,
                  int32_t* status, cudaStream_t s) {
  const int quads = rec_round4(rec.vdim) / 4, cg = quads < kRdThreads ? quads : kRdThreads, rg = kRdThreads / cg;
  const size_t smem = (size_t)(3 * rec_round4(rec.dim) + 3 * rec_round4(rec.vdim) + 8 * rg * cg) * 4;
  if (smem > 200 * 1024) return B200KV_E_RANGE;
  if (cudaFuncSetAttribute(recurrence_decode_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return B200KV_E_LAUNCH;
  return launch_result(launch_chained(recurrence_decode_kernel<T>, dim3(rec.heads, ent.num_entries), dim3(kRdThreads), smem, s, rec, in, ent, norm,
                                      out, cg, rg, status));
}

int recurrence_decode_any(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const b200dec_entries& ent, const RecNorm& norm,
                          void* out, int32_t* status, cudaStream_t s) {
  return rec.elem == 2 ? rd_run<uint16_t>(rec, in, ent, norm, out, status, s) : rd_run<float>(rec, in, ent, norm, out, status, s);
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
  const dim3 grid((ent.num_rows + kRcRun - 1) / kRcRun, ((vec ? rec.channels / 8 : rec.channels) + kRcThreads - 1) / kRcThreads);
  auto* kernel = vec ? (rec.taps == 4   ? conv_rows_kernel<T, 8, 4>
                        : rec.taps == 3 ? conv_rows_kernel<T, 8, 3>
                        : rec.taps == 2 ? conv_rows_kernel<T, 8, 2> : conv_rows_kernel<T, 8, 0>)
                     : conv_rows_kernel<T, 1, 0>;
  return launch_result(launch_chained(kernel, grid, dim3(kRcThreads), 0, s, rec, in, ent, (T*)out, (rec.channels + 7) / 8 * 8, status));
}

}  // namespace b200kv

using namespace b200kv;

extern "C" int b200dec_conv_rows(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const b200dec_entries* ent, void* conv_out,
                                 int32_t* status, void* stream) {
  const int rc = check_recurrence(rec, in, ent);
  if (rc != B200KV_OK) return rc;
  if (!ent->cu_seqlens || !conv_out) return B200KV_E_NULL;
  if (ent->num_rows == 0) return B200KV_OK;
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
