// Prompt portions of the delta rule (one decay per key channel), eight tokens at a time and all in 32-bit.
//
// With L_i the running product of a block's decays up to token i (per key channel), S0 the state in front of the block, and
//   kd_i = k_i * L_i     qd_i = q_i * L_i     kr_j = k_j * (L_8 / L_j)     (quotients as products of the decays between: all <= 1)
//   A_ij = sum_d k_i k_j L_i / L_j  (j < i)     B_ij = sum_d q_i k_j L_i / L_j  (j <= i)
// the block's writes solve a triangular system, u = (I + diag(beta) A)^-1 diag(beta) (v - S0^T kd), the outputs are
// o = S0^T qd + B u, and the state behind is S = L_8 * S0 + sum_j kr_j u_j^T.
//   prepare  one block of threads per (8 tokens, head), all independent: the vectors, the inverse T and B, to a workspace.
//   scan     groups of lanes own four state columns each, block after block: two sums over the key channels per token on the
//            same state, one exchange of the eight tokens' sums between the lanes, the eight writes in one pass.
//            A block's vectors come by bulk copies into a ring; packed 32-bit arithmetic (two rows per instruction).
// Every wait is bounded: when one runs out the block writes nothing more and sets B200KV_S_TIMEOUT.
#include "dec_tma.cuh"
#include "recurrence.cuh"

namespace b200kv {

constexpr int kRbTok = 8;        // tokens per block
constexpr int kRbWarps = 2;      // of a block of the scan
constexpr int kRbCols = 4;       // state columns of a group of lanes
constexpr int kRbStages = 3;

// Workspace of one (block, head) in floats: kd, qd, kr [8][Dp], L_8 [Dp], T [8][8], B [8][8].
__host__ __device__ constexpr int rb_floats(int Dp) { return 3 * kRbTok * Dp + Dp + 2 * kRbTok * kRbTok; }

// First block of entry e in the list of all blocks: never less than the number of blocks of the entries in front.
__device__ __forceinline__ int rb_first(const b200dec_entries& ent, int e) { return ent.cu_seqlens[e] / kRbTok + e; }

// ---------------------------------------------------------------- prepare
constexpr int kRpThreads = 128;
constexpr int kRpSums = 96;  // A (28), B (36), squares of q and of k (8 each), padded for the exchange

__host__ __device__ constexpr int rp_a(int i, int j) { return i * (i - 1) / 2 + j; }       // j < i
__host__ __device__ constexpr int rp_b(int i, int j) { return 28 + i * (i + 1) / 2 + j; }  // j <= i
constexpr int kRpQ = 64, kRpK = 72;

// Sums of 96 values over the warp's lanes; every lane keeps three.
__device__ __forceinline__ void rp_exchange(float (&v)[kRpSums], int lane) {
  int n = kRpSums / 2;
#pragma unroll
  for (int bit = 16; bit > 0; bit >>= 1) {
    const bool hi = lane & bit;
#pragma unroll
    for (int i = 0; i < n; ++i) {
      const float keep = hi ? v[i + n] : v[i], give = hi ? v[i] : v[i + n];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, bit);
    }
    n >>= 1;
  }
}

template <typename T, bool kOne>  // kOne: dim <= kRpThreads, a thread's channel stays in registers
__global__ void __launch_bounds__(kRpThreads)
rb_prepare_kernel(const b200dec_recurrence rec, const b200dec_recurrence_in in, const T* __restrict__ conv, int conv_stride,
                  const b200dec_entries ent, float* __restrict__ ws, int Dp, int32_t* status) {
  __shared__ float red[kRpThreads / 32][kRpSums];
  __shared__ float sums[kRpSums], beta[kRbTok], fq[kRbTok], fk[kRbTok];
  pdl_enter();
  const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
  int lo = 0, hi = ent.num_entries;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (rb_first(ent, mid) <= s) lo = mid; else hi = mid;
  }
  if (lo < *ent.num_decoding) { pdl_wait(); return; }
  const RecEntry x = rec_entry(ent, rec, lo, status);
  const int t0 = (s - rb_first(ent, lo)) * kRbTok, nt = min(kRbTok, x.n - t0);
  pdl_wait();
  if (nt <= 0) return;
  const int D = rec.dim, hq = h / (rec.heads / rec.qk_heads);
  const long long row0 = x.first + t0;
  const float na = rec.neg_a[h];
  const T* steps = (const T*)in.step + row0 * in.step_stride + h * D;
  const T* src = conv + row0 * conv_stride + hq * D;
  if (tid < kRbTok) beta[tid] = tid < nt ? sigmoid_f(ld_elem((const T*)in.beta + (row0 + tid) * in.beta_stride + h)) : 0.f;
  float q[kRbTok], k[kRbTok], g[kRbTok];
  auto load = [&](int d) {
    const float bias = d < D ? rec.dt_bias[h * D + d] : 0.f;
    const T *pq = src + rec.off_q + d, *pk = src + rec.off_k + d, *ps = steps + d;
#pragma unroll
    for (int i = 0; i < kRbTok; ++i) {
      const bool some = i < nt && d < D;
      q[i] = some ? ld_elem(pq) : 0.f;
      k[i] = some ? ld_elem(pk) : 0.f;
      g[i] = some ? ld_elem(ps) + bias : 0.f;
      pq += conv_stride;
      pk += conv_stride;
      ps += in.step_stride;
    }
#pragma unroll
    for (int i = 0; i < kRbTok; ++i) g[i] = i < nt && d < D ? expf(na * softplus_f(g[i])) : 1.f;
  };
  float v[kRpSums];
#pragma unroll
  for (int i = 0; i < kRpSums; ++i) v[i] = 0.f;
  for (int d = tid; d < Dp; d += kRpThreads) {
    load(d);
#pragma unroll
    for (int j = 0; j < kRbTok; ++j) {
      float f = k[j];  // k_j times the decays since
      v[rp_b(j, j)] = fmaf(q[j], f, v[rp_b(j, j)]);
      v[kRpQ + j] = fmaf(q[j], q[j], v[kRpQ + j]);
      v[kRpK + j] = fmaf(f, f, v[kRpK + j]);
#pragma unroll
      for (int i = j + 1; i < kRbTok; ++i) {
        f *= g[i];
        v[rp_a(i, j)] = fmaf(k[i], f, v[rp_a(i, j)]);
        v[rp_b(i, j)] = fmaf(q[i], f, v[rp_b(i, j)]);
      }
    }
  }
  rp_exchange(v, lane);
  {
    const int at = ((lane >> 4) & 1) * 48 + ((lane >> 3) & 1) * 24 + ((lane >> 2) & 1) * 12 + ((lane >> 1) & 1) * 6 + (lane & 1) * 3;
#pragma unroll
    for (int i = 0; i < 3; ++i) red[tid >> 5][at + i] = v[i];
  }
  __syncthreads();
  if (tid < kRpSums) sums[tid] = (red[0][tid] + red[1][tid]) + (red[2][tid] + red[3][tid]);
  __syncthreads();
  if (tid < kRbTok) {
    fq[tid] = rec.q_scale * (rec.unit_norm ? 1.0f / sqrtf(sums[kRpQ + tid] + rec.unit_eps) : 1.f);
    fk[tid] = rec.unit_norm ? 1.0f / sqrtf(sums[kRpK + tid] + rec.unit_eps) : 1.f;
  }
  __syncthreads();
  float* dst = ws + ((long long)s * rec.heads + h) * rb_floats(Dp);
  float* tb = dst + 3 * kRbTok * Dp + Dp;
  for (int d = tid; d < Dp; d += kRpThreads) {
    if (!kOne) load(d);
    float f = 1.f;
#pragma unroll
    for (int i = 0; i < kRbTok; ++i) {
      f *= g[i];
      dst[i * Dp + d] = k[i] * fk[i] * f;
      dst[(kRbTok + i) * Dp + d] = q[i] * fq[i] * f;
    }
    dst[3 * kRbTok * Dp + d] = f;
    f = 1.f;
#pragma unroll
    for (int i = kRbTok - 1; i >= 0; --i) {
      dst[(2 * kRbTok + i) * Dp + d] = k[i] * fk[i] * f;
      f *= g[i];
    }
  }
  if (tid < kRbTok) {  // column tid of the inverse
    float c[kRbTok];
#pragma unroll
    for (int i = 0; i < kRbTok; ++i) {
      float a = i == tid ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) a = fmaf(-sums[rp_a(i, j)] * fk[i] * fk[j], c[j], a);
      c[i] = beta[i] * a;
      tb[i * kRbTok + tid] = c[i];
    }
  } else if (tid >= 64) {
    const int i = (tid - 64) / kRbTok, j = tid % kRbTok;
    tb[kRbTok * kRbTok + tid - 64] = j <= i ? sums[28 + i * (i + 1) / 2 + j] * fq[i] * fk[j] : 0.f;
  }
}

// ---------------------------------------------------------------- scan
typedef unsigned long long rb_pair;  // two 32-bit numbers of neighbouring rows
__device__ __forceinline__ rb_pair rb_pack(float a, float b) {
  rb_pair r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float rb_both(rb_pair p) {
  float a, b;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(p));
  return a + b;
}
__device__ __forceinline__ rb_pair rb_fma(rb_pair a, rb_pair b, rb_pair c) {
  rb_pair r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ rb_pair rb_mul(rb_pair a, rb_pair b) {
  rb_pair r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
// Volatile, so that the loads stay in front of the arithmetic they feed instead of beside it.
__device__ __forceinline__ ulonglong2 rb_lds(uint32_t addr) {
  ulonglong2 v;
  asm volatile("ld.shared.v2.u64 {%0, %1}, [%2];" : "=l"(v.x), "=l"(v.y) : "r"(addr));
  return v;
}
__device__ __forceinline__ void rb_bulk(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

// Sums of 32 values over kLanes lanes, of which each keeps 32 / kLanes: those of token lane / (kLanes / 8) and of columns
// kC * (lane % (kLanes / 8)) on, kC = 32 / kLanes.  A lane holds token i ^ (the token it will keep) in places 4 i .., so that what it gives away in the exchanges over tokens always stands in the same places.
template <int kLanes>
__device__ __forceinline__ void rb_exchange(float (&v)[kRbCols * kRbTok], int lane) {
  int n = kRbCols * kRbTok / 2;
#pragma unroll
  for (int bit = kLanes / 2; bit > 0; bit >>= 1) {
    const bool hi = n < kRbCols && (lane & bit);
#pragma unroll
    for (int i = 0; i < n; ++i) {
      const float keep = hi ? v[i + n] : v[i], give = hi ? v[i] : v[i + n];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, bit);
    }
    n >>= 1;
  }
}

// kLanes lanes share kRbCols state columns; lane l owns rows 4 kLanes j + 4 l + (0..3), j < kR / 4, of all of them.
// One block: kRbWarps warps, 32 kRbCols / kLanes columns each, of one head of one entry.
template <typename T, int kLanes, int kR>
__global__ void __launch_bounds__(32 * kRbWarps)
rb_scan_kernel(const b200dec_recurrence rec, const b200dec_recurrence_in in, const T* __restrict__ conv, int conv_stride,
               const b200dec_entries ent, const float* __restrict__ ws, float* __restrict__ out, int slabs, int32_t* status) {
  constexpr int Dp = kLanes * kR, kFloats = rb_floats(Dp), kQuads = kR / 4, kGroups = 32 / kLanes;
  constexpr int kM = kLanes / 8, kC = kRbCols / kM;  // after the exchange a lane holds kC columns of one token
  extern __shared__ __align__(128) float rb_smem[];  // [kRbStages][kFloats]
  __shared__ __align__(16) float ubuf[kRbWarps][kGroups][kRbTok][kRbCols];
  __shared__ __align__(8) uint64_t bars[kRbStages];
  pdl_enter();
  const int e = blockIdx.y, h = blockIdx.x / slabs, slab = blockIdx.x - h * slabs, tid = threadIdx.x;
  if (e < *ent.num_decoding) { pdl_wait(); return; }
  const RecEntry x = rec_entry(ent, rec, e, status);
  if (tid == 0) {
    for (int i = 0; i < kRbStages; ++i) dt_mbar_init(dt_smem(bars + i), 1);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  __syncthreads();
  pdl_wait();
  if (x.n == 0) return;
  const int D = rec.dim, P = rec.vdim, P4 = rec_round4(P), blocks = (x.n + kRbTok - 1) / kRbTok;
  const int warp = tid >> 5, grp = (tid & 31) / kLanes, l = tid % kLanes;
  const int p0 = ((slab * kRbWarps + warp) * kGroups + grp) * kRbCols;  // the first column
  const int tok = l / kM, pc = p0 + kC * (l % kM);                  // what this lane holds after the exchange
  const long long at0 = (long long)rb_first(ent, e) * rec.heads + h;
  auto fetch = [&](int b) {
    const uint32_t bar = dt_smem(bars + b % kRbStages);
    dt_expect_tx(bar, kFloats * 4);
    rb_bulk(dt_smem(rb_smem + (b % kRbStages) * kFloats), ws + (at0 + (long long)b * rec.heads) * kFloats, kFloats * 4, bar);
  };
  if (tid == 0)
    for (int b = 0; b < min(kRbStages, blocks); ++b) fetch(b);
  float* state = rec.state + ((long long)x.slot * rec.heads + h) * D * P4;
  rb_pair S[kRbCols][kR / 2];  // [column][pair of rows]
#pragma unroll
  for (int i = 0; i < kR / 2; ++i) {
    const int d = (i / 2) * 4 * kLanes + 4 * l + 2 * (i & 1);
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), c = a;
    if (x.pos > 0 && p0 < P4) {
      if (d < D) a = __ldcg(reinterpret_cast<const float4*>(state + (long long)d * P4 + p0));
      if (d + 1 < D) c = __ldcg(reinterpret_cast<const float4*>(state + (long long)(d + 1) * P4 + p0));
    }
    S[0][i] = rb_pack(a.x, c.x);
    S[1][i] = rb_pack(a.y, c.y);
    S[2][i] = rb_pack(a.z, c.z);
    S[3][i] = rb_pack(a.w, c.w);
  }
  // v of this lane's token and columns in block b; kept as loaded until it is used, so that nothing waits for it
  auto value = [&](int b, T (&v)[kC]) {
    const int t = b * kRbTok + tok;
    const T* src = conv + (long long)(x.first + t) * conv_stride + rec.off_v + h * P + pc;
#pragma unroll
    for (int c = 0; c < kC; ++c) v[c] = t < x.n && pc + c < P ? src[c] : T(0);
  };
  T v_next[kC];
  value(0, v_next);
  bool dead = false;
  for (int b = 0; b < blocks; ++b) {
    float w[kC];
#pragma unroll
    for (int c = 0; c < kC; ++c) w[c] = ld_elem(v_next + c);
    value(b + 1, v_next);
    if (!dt_mbar_wait(dt_smem(bars + b % kRbStages), (b / kRbStages) & 1)) dead = true;
    const float* st = rb_smem + (b % kRbStages) * kFloats;
    // this lane's rows of eight vectors (of token i ^ swap in place i), and their sums with the state
    const uint32_t mine = dt_smem(st) + 16 * l;
    auto rows = [&](int vec, int swap, ulonglong2 (&k)[kRbTok][kQuads]) {
#pragma unroll
      for (int i = 0; i < kRbTok; ++i)
#pragma unroll
        for (int j = 0; j < kQuads; ++j) k[i][j] = rb_lds(mine + 4 * ((vec * kRbTok + (i ^ swap)) * Dp + 4 * kLanes * j));
    };
    auto sums = [&](const ulonglong2 (&vec)[kRbTok][kQuads], float (&r)[kRbCols * kRbTok]) {
#pragma unroll
      for (int i = 0; i < kRbTok; ++i) {
        rb_pair acc[kRbCols];
#pragma unroll
        for (int j = 0; j < kQuads; ++j) {
          const ulonglong2 k = vec[i][j];
#pragma unroll
          for (int c = 0; c < kRbCols; ++c) {
            acc[c] = j == 0 ? rb_mul(S[c][0], k.x) : rb_fma(S[c][2 * j], k.x, acc[c]);
            acc[c] = rb_fma(S[c][2 * j + 1], k.y, acc[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < kRbCols; ++c) r[kRbCols * i + c] = rb_both(acc[c]);
      }
    };
    ulonglong2 ka[kRbTok][kQuads], kb[kRbTok][kQuads], decay[kQuads];
    float r[kRbCols * kRbTok], o[kRbCols * kRbTok];
    rows(0, tok, ka);
    rows(1, tok, kb);
    sums(ka, r);
    rows(2, 0, ka);
    rb_exchange<kLanes>(r, l);
    sums(kb, o);
#pragma unroll
    for (int j = 0; j < kQuads; ++j) decay[j] = rb_lds(mine + 4 * (3 * kRbTok * Dp + 4 * kLanes * j));
    rb_exchange<kLanes>(o, l);
    const float* tb = st + 3 * kRbTok * Dp + Dp;
    float row[2][kRbTok];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const float4 a = *reinterpret_cast<const float4*>(tb + (i * kRbTok + tok) * kRbTok);
      const float4 c = *reinterpret_cast<const float4*>(tb + (i * kRbTok + tok) * kRbTok + 4);
      row[i][0] = a.x; row[i][1] = a.y; row[i][2] = a.z; row[i][3] = a.w;
      row[i][4] = c.x; row[i][5] = c.y; row[i][6] = c.z; row[i][7] = c.w;
    }
    float u[kC];
#pragma unroll
    for (int c = 0; c < kC; ++c) {
      w[c] -= r[c];
      float even = 0.f, odd = 0.f;
#pragma unroll
      for (int j = 0; j < kRbTok; ++j) {
        const float wj = __shfl_sync(0xffffffffu, w[c], j * kM + l % kM, kLanes);
        if (j & 1) odd = fmaf(row[0][j], wj, odd); else even = fmaf(row[0][j], wj, even);
      }
      u[c] = even + odd;
      ubuf[warp][grp][tok][kC * (l % kM) + c] = u[c];
    }
    __syncwarp();
    const int t = b * kRbTok + tok;
#pragma unroll
    for (int c = 0; c < kC; ++c) {
      float even = o[c], odd = 0.f;
#pragma unroll
      for (int j = 0; j < kRbTok; ++j) {
        const float uj = ubuf[warp][grp][j][kC * (l % kM) + c];
        if (j & 1) odd = fmaf(row[1][j], uj, odd); else even = fmaf(row[1][j], uj, even);
      }
      if (t < x.n && pc + c < P && !dead) out[((long long)(x.first + t) * rec.heads + h) * P + pc + c] = even + odd;
    }
#pragma unroll
    for (int j = 0; j < kQuads; ++j) {
      const ulonglong2 g = decay[j];
#pragma unroll
      for (int c = 0; c < kRbCols; ++c) {
        S[c][2 * j] = rb_mul(S[c][2 * j], g.x);
        S[c][2 * j + 1] = rb_mul(S[c][2 * j + 1], g.y);
      }
    }
#pragma unroll
    for (int i = 0; i < kRbTok; ++i) {
      const float4 uu = *reinterpret_cast<const float4*>(ubuf[warp][grp][i]);
      const rb_pair up[kRbCols] = {rb_pack(uu.x, uu.x), rb_pack(uu.y, uu.y), rb_pack(uu.z, uu.z), rb_pack(uu.w, uu.w)};
#pragma unroll
      for (int j = 0; j < kQuads; ++j) {
        const ulonglong2 k = ka[i][j];
#pragma unroll
        for (int c = 0; c < kRbCols; ++c) {
          S[c][2 * j] = rb_fma(k.x, up[c], S[c][2 * j]);
          S[c][2 * j + 1] = rb_fma(k.y, up[c], S[c][2 * j + 1]);
        }
      }
    }
    if (__syncthreads_or(dead)) {  // (otherwise: the stage and ubuf are free)
      if (tid == 0) {
        if (status) atomicOr(status, B200KV_S_TIMEOUT);
        for (int i = b; i < min(b + kRbStages, blocks); ++i) dt_mbar_wait(dt_smem(bars + i % kRbStages), (i / kRbStages) & 1);
      }
      __syncthreads();
      return;
    }
    if (tid == 0 && b + kRbStages < blocks) fetch(b + kRbStages);
  }
#pragma unroll
  for (int i = 0; i < kR / 2; ++i) {
    const int d = (i / 2) * 4 * kLanes + 4 * l + 2 * (i & 1);
    float a[kRbCols], c[kRbCols];
#pragma unroll
    for (int k = 0; k < kRbCols; ++k) {
      asm("mov.b64 {%0, %1}, %2;" : "=f"(a[k]), "=f"(c[k]) : "l"(S[k][i]));
      if (p0 + k >= P) a[k] = c[k] = 0.f;
    }
    if (p0 < P4) {
      if (d < D) st_elem4(state + (long long)d * P4 + p0, a);
      if (d + 1 < D) st_elem4(state + (long long)(d + 1) * P4 + p0, c);
    }
  }
  rec_keep_inputs<T>(rec, in, x, blockIdx.x, gridDim.x, 32 * kRbWarps);
}

template <typename T, int kLanes, int kR>
static int rb_launch(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const void* conv, const b200dec_entries& ent, float* ws,
                     float* out, int32_t* status, cudaStream_t s) {
  constexpr int Dp = kLanes * kR, kCols = kRbWarps * 32 / kLanes * kRbCols;
  const int stride = (rec.channels + 7) / 8 * 8, slabs = (rec.vdim + kCols - 1) / kCols;
  const int list = ent.num_rows / kRbTok + ent.num_entries;
  auto* prepare = rec.dim <= kRpThreads ? rb_prepare_kernel<T, true> : rb_prepare_kernel<T, false>;
  const int rc = launch_result(launch_chained(prepare, dim3(list, rec.heads), dim3(kRpThreads), 0, s, rec, in, (const T*)conv, stride, ent, ws, Dp,
                                              status));
  if (rc != B200KV_OK) return rc;
  const size_t smem = (size_t)kRbStages * rb_floats(Dp) * 4;
  if (cudaFuncSetAttribute(rb_scan_kernel<T, kLanes, kR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return B200KV_E_LAUNCH;
  // Not chained: brought up beside the kernel in front, its few long-running blocks would crowd on the multiprocessors that
  // come free first.
  return launch_result(launch_kernel(false, rb_scan_kernel<T, kLanes, kR>, dim3(rec.heads * slabs, ent.num_entries), dim3(32 * kRbWarps), smem, s, rec, in,
                                      (const T*)conv, stride, ent, (const float*)ws, out, slabs, status));
}

template <typename T>
static int rb_run(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const void* conv, const b200dec_entries& ent, float* ws, float* out,
                  int32_t* status, cudaStream_t s) {
  if (rec.dim <= 32) return rb_launch<T, 8, 4>(rec, in, conv, ent, ws, out, status, s);
  if (rec.dim <= 64) return rb_launch<T, 16, 4>(rec, in, conv, ent, ws, out, status, s);
  if (rec.dim <= 128) return rb_launch<T, 16, 8>(rec, in, conv, ent, ws, out, status, s);
  return rb_launch<T, 32, 8>(rec, in, conv, ent, ws, out, status, s);
}

}  // namespace b200kv

using namespace b200kv;

extern "C" size_t b200dec_recurrence_blocked_workspace(const b200dec_recurrence* rec, const b200dec_entries* ent) {
  if (!rec || !ent || !rec->correct || !rec->channel_decay || rec->dim < 1 || rec->dim > 256 || rec->heads < 1) return 0;
  const int Dp = rec->dim <= 32 ? 32 : rec->dim <= 64 ? 64 : rec->dim <= 128 ? 128 : 256;
  return (size_t)(ent->num_rows / kRbTok + ent->num_entries) * rec->heads * rb_floats(Dp) * 4;
}

extern "C" int b200dec_recurrence_blocked(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const void* conv_out,
                                          const b200dec_entries* ent, float* out, void* workspace, size_t workspace_bytes, int32_t* status,
                                          void* stream) {
  const int rc = check_recurrence(rec, in, ent);
  if (rc != B200KV_OK) return rc;
  if (!ent->cu_seqlens || !conv_out || !out || !workspace) return B200KV_E_NULL;
  const size_t need = b200dec_recurrence_blocked_workspace(rec, ent);
  if (need == 0 || rec->heads > 65535 || rec->skip) return B200KV_E_SHAPE;
  if (workspace_bytes < need) return B200KV_E_WORKSPACE;
  if (!aligned(workspace, 128)) return B200KV_E_ALIGN;
  if (ent->num_entries == 0 || ent->num_rows == 0) return B200KV_OK;
  cudaStream_t s = (cudaStream_t)stream;
  return rec->elem == 2 ? rb_run<uint16_t>(*rec, *in, conv_out, *ent, (float*)workspace, out, status, s)
                        : rb_run<float>(*rec, *in, conv_out, *ent, (float*)workspace, out, status, s);
}
