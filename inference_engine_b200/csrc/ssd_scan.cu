// Prompt portions of a state-space layer with one decay per head (bf16 models), sixteen tokens at a time on the tensor cores.
//
// With L_i the sum of a chunk's log-decays up to token i, S0 the state in front of the chunk, b and c the keys and queries:
//   y_i = exp(L_i) S0^T c_i + sum_{j <= i} (c_i . b_j) exp(L_i - L_j) dt_j x_j        S = exp(L_16) S0 + sum_j b_j (dt_j exp(L_16 - L_j) x_j)^T
// One warp owns 16 value columns of a head and keeps S^T [16, state] as the accumulators of bf16 products: as they lie, they
// are the left operand of S^T c, so the state never leaves the registers inside a portion.
// b, c and x are bf16 (the convolution's output).  What is 32-bit enters a product as bf16 terms: the weighted x that is
// written to the state as three, which together carry all 24 bits; the state and the masked scores on their way to an output,
// which leaves here for a bf16 product, as two (17 bits).  Sums are 32-bit, and so is the state.
// A single long portion does not fill the machine.  It is then cut into up to kSsSegments pieces: a first launch carries each
// piece but the last from zero (the first one from the request's state), a second one starts every piece from the pieces in
// front of it, decayed.  How many pieces there are is settled on the device, from the step's entries.
// Chunks arrive by asynchronous copies into a ring shared by a block's warps.
#include "recurrence.cuh"

namespace b200kv {

constexpr int kSsTok = 16;
constexpr int kSsWarps = 4;   // 64 columns per block
constexpr int kSsStages = 4;
constexpr int kSsSegments = 4;
constexpr int kSsMinSegment = 64;  // tokens
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
// a and b as two or three bf16 terms each, which add up to them
__device__ __forceinline__ void ss_split(float a, float b, uint32_t& t0, uint32_t& t1) {
  t0 = ss_pack(a, b);
  t1 = ss_pack(a - ss_lo(t0), b - ss_hi(t0));
}
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

// The pieces entry e is cut into: `count` of `len` tokens (the last one shorter).  Workspace places: first .. for the ends
// of pieces, front for the state the entry came with.
struct SsCut {
  int count, len, first, front;
};
__device__ __forceinline__ SsCut ss_cut(const b200dec_entries& ent, int nd, int e, int n, int max_segments, int lane) {
  SsCut c{1, n, 0, 0};
  if (max_segments < 2) return c;
  int live = 0, before = 0;  // entries with a portion, and those in front of e
  for (int i = nd + lane; i < ent.num_entries; i += 32) {
    const bool some = ent.cu_seqlens[i + 1] > ent.cu_seqlens[i] && ent.slots[i] >= 0;
    live += some;
    before += some && i < e;
  }
  live = __reduce_add_sync(0xffffffffu, live);
  before = __reduce_add_sync(0xffffffffu, before);
  c.count = max(1, min(max_segments / max(live, 1), n / kSsMinSegment));
  c.len = ((n + c.count - 1) / c.count + kSsTok - 1) / kSsTok * kSsTok;
  c.count = (n + c.len - 1) / c.len;
  c.first = before * (max_segments / max(live, 1));
  c.front = kSsSegments + before;  // there are places for every entry that is cut: it is one of at most max_segments / 2
  return c;
}

// kN16: 16-channel pieces of the state's rows (padding is zero).  kLocal: the first launch.
// Workspace: 2 * kSsSegments places of [head][state channel][round4(vdim)], then [kSsSegments][head] sums of log-decays.
template <int kN16, bool kLocal>
__global__ void __launch_bounds__(32 * kSsWarps)
ssd_scan_kernel(const b200dec_recurrence rec, const b200dec_recurrence_in in, const uint16_t* __restrict__ conv, int conv_stride,
                const b200dec_entries ent, float* __restrict__ out, int slabs, int max_segments, float* ws, int32_t* status) {
  constexpr int kN = 16 * kN16, kRow = kN + 8;  // bf16 per row of b and c in shared memory
  constexpr uint32_t kStage = kSsTok * (2 * kRow + kSsXRow) * 2;
  extern __shared__ __align__(16) uint8_t ss_smem[];
  pdl_enter();
  const int e = blockIdx.y, h = blockIdx.x / slabs, slab = blockIdx.x - h * slabs, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int seg = blockIdx.z, nd = *ent.num_decoding;
  if (e < nd) { pdl_wait(); return; }
  const RecEntry all = rec_entry(ent, rec, e, status);
  const SsCut cut = ss_cut(ent, nd, e, all.n, max_segments, lane);
  pdl_wait();
  if (all.n == 0 || seg >= cut.count || (kLocal && seg >= cut.count - 1)) return;
  RecEntry x = all;  // this piece
  x.first += seg * cut.len;
  x.n = min(cut.len, all.n - seg * cut.len);
  const int N = rec.dim, P = rec.vdim, P4 = rec_round4(P), grp = h / (rec.heads / rec.qk_heads);
  const int chunks = (x.n + kSsTok - 1) / kSsTok, col0 = slab * 16 * kSsWarps;
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(ss_smem);
  // this thread's 16-byte pieces of a chunk (rows of c | b | x; zero behind the portion and behind the sizes)
  constexpr int kPer = 2 * (kN / 8) + 2 * kSsWarps, kItems = (kSsTok * kPer + 32 * kSsWarps - 1) / (32 * kSsWarps);
  int src_off[kItems];  // elements from the chunk's first row, -1: nothing there
  uint32_t dst_off[kItems];
#pragma unroll
  for (int q = 0; q < kItems; ++q) {
    const int i = tid + q * 32 * kSsWarps, r = i / kPer, k = i - r * kPer;
    int ch = -1;
    if (k < kN / 8) {
      if (8 * k < N) ch = rec.off_q + grp * N + 8 * k;
      dst_off[q] = r * kRow * 2 + 16 * k;
    } else if (k < 2 * (kN / 8)) {
      const int m = k - kN / 8;
      if (8 * m < N) ch = rec.off_k + grp * N + 8 * m;
      dst_off[q] = (kSsTok + r) * kRow * 2 + 16 * m;
    } else {
      const int m = k - 2 * (kN / 8);
      if (col0 + 8 * m < P) ch = rec.off_v + h * P + col0 + 8 * m;
      dst_off[q] = 2 * kSsTok * kRow * 2 + r * kSsXRow * 2 + 16 * m;
    }
    src_off[q] = r >= kSsTok ? -2 : (ch < 0 ? -1 : r * conv_stride + ch);
  }
  auto fetch = [&](int c) {
    if (c < chunks) {
      const uint32_t st = base + (c % kSsStages) * kStage;
      const uint16_t* rows = conv + (long long)(x.first + c * kSsTok) * conv_stride;
      const int end = (x.n - c * kSsTok) * conv_stride;  // rows behind the piece start here
#pragma unroll
      for (int q = 0; q < kItems; ++q)
        if (src_off[q] != -2) {
          const bool ok = src_off[q] >= 0 && src_off[q] < end;
          ss_cp16(st + dst_off[q], ok ? rows + src_off[q] : conv, ok ? 16 : 0);
        }
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  const int g = lane >> 2, t2 = 2 * (lane & 3), m8 = lane >> 3, r8 = lane & 7;
  const int p0 = col0 + warp * 16 + g;  // this lane's rows of S^T: p0 and p0 + 8
  const long long head_floats = (long long)N * P4;
  float* state = rec.state + ((long long)x.slot * rec.heads + h) * head_floats;
  auto place = [&](int i) { return ws + ((long long)i * rec.heads + h) * head_floats; };
  float* logs = ws + 2 * kSsSegments * rec.heads * head_floats;
  float S[2 * kN16][4];
  auto each = [&](auto f) {  // over the state entries this lane holds
#pragma unroll
    for (int n = 0; n < 2 * kN16; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) f(S[n][i], 8 * n + t2 + (i & 1), p0 + 4 * (i & 2));
  };
  auto take = [&](const float* src) {
    each([&](float& s, int d, int p) { s = d < N && p < P ? __ldcg(src + (long long)d * P4 + p) : 0.f; });
  };
  auto put = [&](float* dst) {
    each([&](float& s, int d, int p) { if (d < N && p < P4) dst[(long long)d * P4 + p] = p < P ? s : 0.f; });
  };
  each([&](float& s, int, int) { s = 0.f; });
  if (kLocal) {
    if (seg == 0) {
      if (x.pos > 0) take(state);
      put(place(cut.front));
    }
  } else if (cut.count == 1) {
    if (x.pos > 0) take(state);
  } else if (seg == 0) {
    take(place(cut.front));
  } else {
    take(place(cut.first));
    for (int r = 1; r < seg; ++r) {
      const float f = exp2f(__ldcg(logs + (long long)(cut.first + r) * rec.heads + h));
      const float* src = place(cut.first + r);
      each([&](float& s, int d, int p) { s = fmaf(s, f, d < N && p < P ? __ldcg(src + (long long)d * P4 + p) : 0.f); });
    }
  }
  const float na = rec.neg_a[h] * 1.4426950408889634f, bias = rec.dt_bias[h], skip = rec.skip ? rec.skip[h] : 0.f;
  auto raw_step = [&](int c) {
    const int t = c * kSsTok + (lane & 15);
    return t < x.n ? ld_elem((const uint16_t*)in.step + (long long)(x.first + t) * in.step_stride + h) : 0.f;
  };
  float raw = raw_step(0), log_sum = 0.f;
  for (int c = 0; c < kSsStages - 1; ++c) fetch(c);
  for (int c = 0; c < chunks; ++c) {
    asm volatile("cp.async.wait_group %0;\n" ::"n"(kSsStages - 2) : "memory");
    __syncthreads();  // the chunk is there for every warp, and the stage of the one before is free
    fetch(c + kSsStages - 1);
    // ---- steps and log-decays of the sixteen tokens (lanes 16.. repeat them)
    const float dt = c * kSsTok + (lane & 15) < x.n ? softplus_f(raw + bias) : 0.f;
    raw = raw_step(c + 1);
    float L = na * dt;  // in units of log 2
#pragma unroll
    for (int o = 1; o < kSsTok; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, L, o, 16);
      if ((lane & 15) >= o) L += v;
    }
    const float total = __shfl_sync(0xffffffffu, L, 15);
    log_sum += total;
    float Lj[4], dtj[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int j = t2 + (i & 1) + 4 * (i & 2);  // tokens t2, t2 + 1, t2 + 8, t2 + 9
      Lj[i] = __shfl_sync(0xffffffffu, L, j);
      dtj[i] = __shfl_sync(0xffffffffu, dt, j);
    }
    const float Li[2] = {__shfl_sync(0xffffffffu, L, g), __shfl_sync(0xffffffffu, L, g + 8)};
    const uint32_t sc = base + (c % kSsStages) * kStage, sb = sc + kSsTok * kRow * 2, sx = sb + kSsTok * kRow * 2;
    uint32_t fx[4];
    ss_ldsm_t(fx, sx + ((m8 >> 1) * 8 + r8) * kSsXRow * 2 + (warp * 16 + (m8 & 1) * 8) * 2);
    if constexpr (!kLocal) {
      // ---- c . b of all pairs of tokens, and S0^T c
      float cb[2][4] = {}, y[2][2][4] = {};
#pragma unroll
      for (int k = 0; k < kN16; ++k) {
        const uint32_t off = ((m8 & 1) * 8 + r8) * kRow * 2 + (16 * k + (m8 >> 1) * 8) * 2;
        uint32_t fc[4], fb[4], a[2][4];
        ss_ldsm(fc, sc + off);
        ss_ldsm(fb, sb + off);
        ss_mma(cb[0], fc, fb[0], fb[2]);
        ss_mma(cb[1], fc, fb[1], fb[3]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float* s = S[2 * k + (i >> 1)];
          ss_split(s[2 * (i & 1)], s[2 * (i & 1) + 1], a[0][i], a[1][i]);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          ss_mma(y[i][0], a[i], fc[0], fc[2]);
          ss_mma(y[i][1], a[i], fc[1], fc[3]);
        }
      }
      float Y[2][4], ej[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) ej[i] = exp2f(Lj[i]);
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) Y[n][i] = (y[0][n][i] + y[1][n][i]) * ej[2 * n + (i & 1)];
      // ---- tokens of the chunk: x^T times the masked, decayed scores
      uint32_t mt[2][2][2];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int b = 0; b < 2; ++b) {  // row i = g + 8 n, tokens j = t2 + 8 b, + 1
          float m[2];
#pragma unroll
          for (int u = 0; u < 2; ++u) m[u] = t2 + 8 * b + u <= g + 8 * n ? cb[b][2 * n + u] * exp2f(Li[n] - Lj[2 * b + u]) * dtj[2 * b + u] : 0.f;
          ss_split(m[0], m[1], mt[n][b][0], mt[n][b][1]);
        }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
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
    }
    // ---- the state behind the chunk
    uint32_t xs[3][4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int j = 2 * (i >> 1);
      const float w0 = dtj[j] * exp2f(total - Lj[j]), w1 = dtj[j + 1] * exp2f(total - Lj[j + 1]);
      ss_split(ss_lo(fx[i]) * w0, ss_hi(fx[i]) * w1, xs[0][i], xs[1][i], xs[2][i]);
    }
    const float decay = exp2f(total);
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
  if (kLocal) {
    put(place(cut.first + seg));
    if (tid == 0 && slab == 0) logs[(long long)(cut.first + seg) * rec.heads + h] = log_sum;
  } else if (seg == cut.count - 1) {
    put(state);
    rec_keep_inputs<uint16_t>(rec, in, all, blockIdx.x, gridDim.x, 32 * kSsWarps);
  }
}

// Pieces of a portion a launch makes room for: as many as two blocks per multiprocessor allow.
static int ss_segments(const b200dec_recurrence& rec, int sm_count) {
  const int blocks = rec.heads * ((rec.vdim + 16 * kSsWarps - 1) / (16 * kSsWarps)), fit = 2 * sm_count / blocks;
  return fit < 2 ? 1 : (fit < kSsSegments ? fit : kSsSegments);
}

template <int kN16>
static int ss_launch(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const void* conv, const b200dec_entries& ent, float* out,
                     float* ws, int max_segments, int32_t* status, cudaStream_t s) {
  const int slabs = (rec.vdim + 16 * kSsWarps - 1) / (16 * kSsWarps), stride = (rec.channels + 7) / 8 * 8;
  const size_t smem = (size_t)kSsStages * kSsTok * (2 * (16 * kN16 + 8) + kSsXRow) * 2;
  if (cudaFuncSetAttribute(ssd_scan_kernel<kN16, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess ||
      cudaFuncSetAttribute(ssd_scan_kernel<kN16, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return B200KV_E_LAUNCH;
  if (max_segments > 1 && ent.num_rows >= 2 * kSsMinSegment) {
    const int rc = launch_result(launch_chained(ssd_scan_kernel<kN16, true>, dim3(rec.heads * slabs, ent.num_entries, max_segments - 1),
                                                dim3(32 * kSsWarps), smem, s, rec, in, (const uint16_t*)conv, stride, ent, out, slabs,
                                                max_segments, ws, status));
    if (rc != B200KV_OK) return rc;
  } else {
    max_segments = 1;
  }
  return launch_result(launch_chained(ssd_scan_kernel<kN16, false>, dim3(rec.heads * slabs, ent.num_entries, max_segments), dim3(32 * kSsWarps),
                                      smem, s, rec, in, (const uint16_t*)conv, stride, ent, out, slabs, max_segments, ws, status));
}

}  // namespace b200kv

using namespace b200kv;

static bool ss_applies(const b200dec_recurrence* r) {
  return r && r->elem == 2 && !r->correct && !r->channel_decay && !r->unit_norm && r->q_scale == 1.f && r->dim >= 1 && r->dim <= 128 &&
         r->dim % 8 == 0 && r->vdim % 8 == 0 && r->off_q % 8 == 0 && r->off_k % 8 == 0 && r->off_v % 8 == 0;
}

extern "C" size_t b200dec_state_space_chunked_workspace(const b200dec_recurrence* r) {
  if (!ss_applies(r)) return 0;
  return ((size_t)2 * kSsSegments * r->heads * r->dim * rec_round4(r->vdim) + (size_t)kSsSegments * r->heads) * 4;
}

extern "C" int b200dec_state_space_chunked(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const void* conv_out,
                                           const b200dec_entries* ent, float* out, void* workspace, size_t workspace_bytes, int32_t sm_count,
                                           int32_t* status, void* stream) {
  const int rc = check_recurrence(rec, in, ent);
  if (rc != B200KV_OK) return rc;
  if (!ent->cu_seqlens || !conv_out || !out || !workspace) return B200KV_E_NULL;
  if (!ss_applies(rec) || sm_count < 1) return B200KV_E_SHAPE;
  if (workspace_bytes < b200dec_state_space_chunked_workspace(rec)) return B200KV_E_WORKSPACE;
  if ((long long)(rec->channels + 7) * (kSsTok + 1) > 0x7FFFFFFFll || (long long)ent->num_rows * (rec->channels + 7) > 0x7FFFFFFFll)
    return B200KV_E_RANGE;
  if (!aligned(conv_out, 16) || !aligned(workspace, 16)) return B200KV_E_ALIGN;
  if (ent->num_entries == 0 || ent->num_rows == 0) return B200KV_OK;
  cudaStream_t s = (cudaStream_t)stream;
  float* ws = (float*)workspace;
  const int m = ss_segments(*rec, sm_count);
  if (rec->dim <= 16) return ss_launch<1>(*rec, *in, conv_out, *ent, out, ws, m, status, s);
  if (rec->dim <= 32) return ss_launch<2>(*rec, *in, conv_out, *ent, out, ws, m, status, s);
  if (rec->dim <= 64) return ss_launch<4>(*rec, *in, conv_out, *ent, out, ws, m, status, s);
  return ss_launch<8>(*rec, *in, conv_out, *ent, out, ws, m, status, s);
}
