// Prompt portions of a state-space layer with one decay per head (bf16 models), sixteen tokens at a time on the tensor cores.
//
// With L_i the sum of a chunk's log-decays up to token i, S0 the state in front of the chunk, b and c the keys and queries:
//   y_i = exp(L_i) S0^T c_i + sum_{j <= i} (c_i . b_j) exp(L_i - L_j) dt_j x_j        S = exp(L_16) S0 + sum_j b_j (dt_j exp(L_16 - L_j) x_j)^T
// One warp owns 16 value columns of a head and keeps S^T [16, state] as the accumulators of bf16 products: as they lie, they
// are the left operand of S^T c, so the state never leaves the registers inside a portion.
// b, c and x are bf16 (the convolution's output).  What is 32-bit - the state, the masked score matrix, the weighted x - enters
// a product as three bf16 terms, which together carry all 24 bits, and sums are 32-bit.
// Chunks arrive by asynchronous copies into a ring shared by a block's warps.
#include "recurrence.cuh"

namespace b200kv {

constexpr int kSsTok = 16;
constexpr int kSsWarps = 4;   // 64 columns per block
constexpr int kSsStages = 4;
constexpr int kSsXRow = 16 * kSsWarps + 8;  // bf16 per row of x in shared memory (the padding spreads rows over the banks)

__device__ __forceinline__ void ss_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ss_ldsm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ss_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ uint32_t ss_pack(float lo, float hi) {
  uint32_t r;
  asm("cvt.rn.bf16x2.f32 %0, %1, %2;\n" : "=r"(r) : "f"(hi), "f"(lo));
  return r;
}
__device__ __forceinline__ float ss_lo(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float ss_hi(uint32_t v) { return __uint_as_float(v & 0xFFFF0000u); }
// a and b as three bf16 terms each: t[0] + t[1] + t[2]
__device__ __forceinline__ void ss_split(float a, float b, uint32_t& t0, uint32_t& t1, uint32_t& t2) {
  t0 = ss_pack(a, b);
  a -= ss_lo(t0);
  b -= ss_hi(t0);
  t1 = ss_pack(a, b);
  t2 = ss_pack(a - ss_lo(t1), b - ss_hi(t1));
}
__device__ __forceinline__ void ss_cp16(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}

template <int kN16>  // 16-channel pieces of the state's rows (padding is zero)
__global__ void __launch_bounds__(32 * kSsWarps)
ssd_scan_kernel(const b200dec_recurrence rec, const b200dec_recurrence_in in, const uint16_t* __restrict__ conv, int conv_stride,
                const b200dec_entries ent, float* __restrict__ out, int slabs, int32_t* status) {
  constexpr int kN = 16 * kN16, kRow = kN + 8;  // bf16 per row of b and c in shared memory
  constexpr uint32_t kStage = kSsTok * (2 * kRow + kSsXRow) * 2;
  extern __shared__ __align__(16) uint8_t ss_smem[];
  pdl_enter();
  const int e = blockIdx.y, h = blockIdx.x / slabs, slab = blockIdx.x - h * slabs, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (e < *ent.num_decoding) { pdl_wait(); return; }
  const RecEntry x = rec_entry(ent, rec, e, status);
  pdl_wait();
  if (x.n == 0) return;
  const int N = rec.dim, P = rec.vdim, P4 = rec_round4(P), grp = h / (rec.heads / rec.qk_heads);
  const int chunks = (x.n + kSsTok - 1) / kSsTok, col0 = slab * 16 * kSsWarps;
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(ss_smem);
  auto fetch = [&](int c) {  // chunk c: rows of c | b | x, zero behind the portion and behind the sizes
    if (c < chunks) {
      const uint32_t st = base + (c % kSsStages) * kStage;
      constexpr int kPer = 2 * (kN / 8) + 2 * kSsWarps;
      for (int i = tid; i < kSsTok * kPer; i += 32 * kSsWarps) {
        const int r = i / kPer, k = i - r * kPer, t = c * kSsTok + r;
        const uint16_t* src = conv + (long long)(x.first + min(t, x.n - 1)) * conv_stride;
        uint32_t dst = st + r * kRow * 2;
        bool in_row;
        if (k < kN / 8) {
          in_row = 8 * k < N;
          src += rec.off_q + grp * N + 8 * k;
          dst += 16 * k;
        } else if (k < 2 * (kN / 8)) {
          const int m = k - kN / 8;
          in_row = 8 * m < N;
          src += rec.off_k + grp * N + 8 * m;
          dst += kSsTok * kRow * 2 + 16 * m;
        } else {
          const int m = k - 2 * (kN / 8);
          in_row = col0 + 8 * m < P;
          src += rec.off_v + h * P + col0 + 8 * m;
          dst = st + 2 * kSsTok * kRow * 2 + r * kSsXRow * 2 + 16 * m;
        }
        const bool ok = in_row && t < x.n;
        ss_cp16(dst, ok ? src : conv, ok ? 16 : 0);
      }
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  const int g = lane >> 2, t2 = 2 * (lane & 3), m8 = lane >> 3, r8 = lane & 7;
  const int p0 = col0 + warp * 16 + g;  // this lane's rows of S^T: p0 and p0 + 8
  float* state = rec.state + ((long long)x.slot * rec.heads + h) * N * P4;
  float S[2 * kN16][4];
#pragma unroll
  for (int n = 0; n < 2 * kN16; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = 8 * n + t2 + (i & 1), p = p0 + 4 * (i & 2);
      S[n][i] = x.pos > 0 && d < N && p < P ? __ldcg(state + (long long)d * P4 + p) : 0.f;
    }
  const float na = rec.neg_a[h], bias = rec.dt_bias[h], skip = rec.skip ? rec.skip[h] : 0.f;
  auto raw_step = [&](int c) {
    const int t = c * kSsTok + (lane & 15);
    return t < x.n ? ld_elem((const uint16_t*)in.step + (long long)(x.first + t) * in.step_stride + h) : 0.f;
  };
  float raw = raw_step(0);
  for (int c = 0; c < kSsStages - 1; ++c) fetch(c);
  for (int c = 0; c < chunks; ++c) {
    asm volatile("cp.async.wait_group %0;\n" ::"n"(kSsStages - 2) : "memory");
    __syncthreads();  // the chunk is there for every warp, and the stage of the one before is free
    fetch(c + kSsStages - 1);
    // ---- steps and log-decays of the sixteen tokens (lanes 16.. repeat them)
    const float dt = c * kSsTok + (lane & 15) < x.n ? softplus_f(raw + bias) : 0.f;
    raw = raw_step(c + 1);
    float L = na * dt;
#pragma unroll
    for (int o = 1; o < kSsTok; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, L, o, 16);
      if ((lane & 15) >= o) L += v;
    }
    const float total = __shfl_sync(0xffffffffu, L, 15);
    float Lj[4], dtj[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int j = t2 + (i & 1) + 4 * (i & 2);  // tokens t2, t2 + 1, t2 + 8, t2 + 9
      Lj[i] = __shfl_sync(0xffffffffu, L, j);
      dtj[i] = __shfl_sync(0xffffffffu, dt, j);
    }
    const float Li[2] = {__shfl_sync(0xffffffffu, L, g), __shfl_sync(0xffffffffu, L, g + 8)};
    const uint32_t sc = base + (c % kSsStages) * kStage, sb = sc + kSsTok * kRow * 2, sx = sb + kSsTok * kRow * 2;
    // ---- c . b of all pairs of tokens, and S0^T c
    float cb[2][4] = {}, y[3][2][4] = {};
#pragma unroll
    for (int k = 0; k < kN16; ++k) {
      const uint32_t off = ((m8 & 1) * 8 + r8) * kRow * 2 + (16 * k + (m8 >> 1) * 8) * 2;
      uint32_t fc[4], fb[4], a[3][4];
      ss_ldsm(fc, sc + off);
      ss_ldsm(fb, sb + off);
      ss_mma(cb[0], fc, fb[0], fb[2]);
      ss_mma(cb[1], fc, fb[1], fb[3]);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float* s = S[2 * k + (i >> 1)];
        ss_split(s[2 * (i & 1)], s[2 * (i & 1) + 1], a[0][i], a[1][i], a[2][i]);
      }
#pragma unroll
      for (int i = 0; i < 3; ++i) {
        ss_mma(y[i][0], a[i], fc[0], fc[2]);
        ss_mma(y[i][1], a[i], fc[1], fc[3]);
      }
    }
    float Y[2][4], ej[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) ej[i] = expf(Lj[i]);
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) Y[n][i] = (y[0][n][i] + (y[1][n][i] + y[2][n][i])) * ej[2 * n + (i & 1)];
    // ---- tokens of the chunk: x^T times the masked, decayed scores
    uint32_t fx[4], mt[2][2][3];
    ss_ldsm_t(fx, sx + ((m8 >> 1) * 8 + r8) * kSsXRow * 2 + (warp * 16 + (m8 & 1) * 8) * 2);
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int b = 0; b < 2; ++b) {  // row i = g + 8 n, tokens j = t2 + 8 b, + 1
        float m[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) m[u] = t2 + 8 * b + u <= g + 8 * n ? cb[b][2 * n + u] * expf(Li[n] - Lj[2 * b + u]) * dtj[2 * b + u] : 0.f;
        ss_split(m[0], m[1], mt[n][b][0], mt[n][b][1], mt[n][b][2]);
      }
#pragma unroll
    for (int i = 0; i < 3; ++i) {
      ss_mma(Y[0], fx, mt[0][0][i], mt[0][1][i]);
      ss_mma(Y[1], fx, mt[1][0][i], mt[1][1][i]);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const uint32_t xv = fx[2 * n + (i >> 1)];
        const int t = c * kSsTok + 8 * n + t2 + (i & 1), p = p0 + 4 * (i & 2);
        const float o = fmaf(skip, i & 1 ? ss_hi(xv) : ss_lo(xv), Y[n][i]);
        if (t < x.n && p < P) out[((long long)(x.first + t) * rec.heads + h) * P + p] = o;
      }
    // ---- the state behind the chunk
    uint32_t xs[3][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int j = 2 * (i >> 1);
      const float w0 = dtj[j] * expf(total - Lj[j]), w1 = dtj[j + 1] * expf(total - Lj[j + 1]);
      ss_split(ss_lo(fx[i]) * w0, ss_hi(fx[i]) * w1, xs[0][i], xs[1][i], xs[2][i]);
    }
    const float decay = expf(total);
#pragma unroll
    for (int k = 0; k < kN16; ++k) {
      uint32_t fb[4];
      ss_ldsm_t(fb, sb + ((m8 & 1) * 8 + r8) * kRow * 2 + (16 * k + (m8 >> 1) * 8) * 2);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        S[2 * k][i] *= decay;
        S[2 * k + 1][i] *= decay;
      }
#pragma unroll
      for (int i = 0; i < 3; ++i) {
        ss_mma(S[2 * k], xs[i], fb[0], fb[1]);
        ss_mma(S[2 * k + 1], xs[i], fb[2], fb[3]);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;\n" ::: "memory");
#pragma unroll
  for (int n = 0; n < 2 * kN16; ++n)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = 8 * n + t2 + (i & 1), p = p0 + 4 * (i & 2);
      if (d < N && p < P4) state[(long long)d * P4 + p] = p < P ? S[n][i] : 0.f;
    }
  rec_keep_inputs<uint16_t>(rec, in, x, blockIdx.x, gridDim.x, 32 * kSsWarps);
}

template <int kN16>
static int ss_launch(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const void* conv, const b200dec_entries& ent, float* out,
                     int32_t* status, cudaStream_t s) {
  const int slabs = (rec.vdim + 16 * kSsWarps - 1) / (16 * kSsWarps);
  const size_t smem = (size_t)kSsStages * kSsTok * (2 * (16 * kN16 + 8) + kSsXRow) * 2;
  if (cudaFuncSetAttribute(ssd_scan_kernel<kN16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return B200KV_E_LAUNCH;
  return launch_result(launch_chained(ssd_scan_kernel<kN16>, dim3(rec.heads * slabs, ent.num_entries), dim3(32 * kSsWarps), smem, s, rec, in,
                                      (const uint16_t*)conv, (rec.channels + 7) / 8 * 8, ent, out, slabs, status));
}

}  // namespace b200kv

using namespace b200kv;

extern "C" int b200dec_state_space_chunked_applies(const b200dec_recurrence* r) {
  return r && r->elem == 2 && !r->correct && !r->channel_decay && !r->unit_norm && r->q_scale == 1.f && r->dim <= 128 && r->dim % 8 == 0 &&
         r->vdim % 8 == 0 && r->off_q % 8 == 0 && r->off_k % 8 == 0 && r->off_v % 8 == 0;
}

extern "C" int b200dec_state_space_chunked(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const void* conv_out,
                                           const b200dec_entries* ent, float* out, int32_t* status, void* stream) {
  const int rc = check_recurrence(rec, in, ent);
  if (rc != B200KV_OK) return rc;
  if (!ent->cu_seqlens || !conv_out || !out) return B200KV_E_NULL;
  if (!b200dec_state_space_chunked_applies(rec)) return B200KV_E_SHAPE;
  if (!aligned(conv_out, 16)) return B200KV_E_ALIGN;
  if (ent->num_entries == 0 || ent->num_rows == 0) return B200KV_OK;
  cudaStream_t s = (cudaStream_t)stream;
  if (rec->dim <= 16) return ss_launch<1>(*rec, *in, conv_out, *ent, out, status, s);
  if (rec->dim <= 32) return ss_launch<2>(*rec, *in, conv_out, *ent, out, status, s);
  if (rec->dim <= 64) return ss_launch<4>(*rec, *in, conv_out, *ent, out, status, s);
  return ss_launch<8>(*rec, *in, conv_out, *ent, out, status, s);
}
