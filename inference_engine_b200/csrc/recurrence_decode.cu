// Decoding entries of a recurrent layer (recurrence.cu has the mathematics and the form for states of any size): a persistent
// grid whose blocks walk through (entry, head) items.  HBM-bound: a state is read once and written once.
// States come and go by bulk copies through a ring in shared memory, two items ahead of the arithmetic; the item's few
// channels (convolution inputs and weights, steps) are gathered into registers one item ahead, and the position and slot that
// takes two items ahead.  One item: convolution and silu,
// norms and decays, (decay S)^T k and (decay S)^T q over all rows, the write, the read-out and optionally its gated norm.
// Every wait is bounded: when one runs out the block stops, lets its copies land and sets B200KV_S_TIMEOUT.
#include "dec_tma.cuh"
#include "recurrence.cuh"

namespace b200kv {

constexpr int kRpdTaps = 4;   // more taps: the other form
constexpr int kRpdStages = 3;

__device__ __forceinline__ void rpd_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];\n"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}
__device__ __forceinline__ void rpd_store(void* dst, uint32_t src, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;\n" ::"l"(dst), "r"(src), "r"(bytes) : "memory");
  asm volatile("cp.async.bulk.commit_group;\n" ::: "memory");
}

// Two neighbouring columns per instruction.
typedef unsigned long long rpd_pair;
__device__ __forceinline__ rpd_pair rpd_both(float a) {
  rpd_pair r;
  asm("mov.b64 %0, {%1, %1};" : "=l"(r) : "f"(a));
  return r;
}
__device__ __forceinline__ rpd_pair rpd_mul(rpd_pair a, rpd_pair b) {
  rpd_pair r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ rpd_pair rpd_fma(rpd_pair a, rpd_pair b, rpd_pair c) {
  rpd_pair r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}

// What an item needs beside its state: up to two channels per thread of q | k | v (dim, dim, vdim of them).  The items of a
// group of heads follow one another; all but the first find q and k where the one before left them.
template <typename T>
struct RpdItem {
  T raw[2], past[2][kRpdTaps - 1], step, beta, gate;  // step: of key channel tid, or of the head
  float w[2][kRpdTaps], bias[2], dt_bias, neg_a, skip;
  int k[2];       // which of the q | k | v channels (-1: none)
  int at;         // the token's place in the ring
  bool same;      // q and k are there already
  bool fresh;     // the state starts here
  bool ok;
  int row, head, slot;  // row: also the entry, since decoding entries come first with one row each
};

template <typename T, int kRows, int kRpdThreads>  // kRows: rows of the state per thread
__global__ void __launch_bounds__(kRpdThreads, kRows > 8 ? 1 : 512 / kRpdThreads)
recurrence_step_kernel(const b200dec_recurrence rec, const b200dec_recurrence_in in, const b200dec_entries ent, const RecNorm norm,
                       void* __restrict__ out, int cg, int rg, int32_t* status) {
  extern __shared__ __align__(128) float rpd_smem[];
  __shared__ float part[4][kRpdThreads / 32];  // squares of q, of k, q . k, squares of the output
  __shared__ __align__(8) uint64_t bars[kRpdStages];
  pdl_enter();
  const int tid = threadIdx.x, D = rec.dim, P = rec.vdim, P4 = rec_round4(P), Dp = rec_round4(D), H = rec.heads;
  const int floats = D * P4;
  const uint32_t bytes = (uint32_t)floats * 4;
  float* qs = rpd_smem + kRpdStages * ((floats + 31) / 32 * 32);
  float *ks = qs + Dp, *gs = ks + Dp, *vs = gs + Dp, *us = vs + P4, *os = us + P4, *red = os + P4;
  auto stage = [&](int i) { return rpd_smem + (i % kRpdStages) * ((floats + 31) / 32 * 32); };
  const int nd = max(0, min(*ent.num_decoding, ent.num_entries));
  const int items = nd * H, share = (items + (int)gridDim.x - 1) / (int)gridDim.x;
  const int i0 = blockIdx.x * share, n = min(share, items - i0);
  if (tid == 0) {
    for (int i = 0; i < kRpdStages; ++i) dt_mbar_init(dt_smem(bars + i), 1);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  __syncthreads();
  pdl_wait();
  if (!ent.cu_seqlens) {  // pure decode: idle rows are cleared
    const int row = H * P;
    for (int r = nd + blockIdx.x; r < min(ent.num_entries, ent.num_rows); r += gridDim.x)
      for (int p = tid; p < row; p += kRpdThreads) {
        if (norm.weight) st_elem((T*)out + r * norm.out_stride + p, 0.f);
        else ((float*)out)[(long long)r * row + p] = 0.f;
      }
  }
  if (n <= 0) return;
  const int per = H / rec.qk_heads;
  auto channel = [&](int k, int h) {  // convolution channel of the k-th of a head's q | k | v channels
    return k < D ? rec.off_q + h / per * D + k : k < 2 * D ? rec.off_k + h / per * D + k - D : rec.off_v + h * P + k - 2 * D;
  };
  auto state_of = [&](int slot, int h) { return rec.state + ((long long)slot * H + h) * floats; };
  auto fetch = [&](int i) {  // by one thread; an arrival without a copy where there is nothing to read
    const int e = (i0 + i) / H, h = (i0 + i) - e * H, slot = ent.slots[e];
    const uint32_t bar = dt_smem(bars + i % kRpdStages);
    if (slot >= 0 && slot < rec.num_slots && ent.cached_lens[e] > 0) {
      dt_expect_tx(bar, bytes);
      rpd_load(dt_smem(stage(i)), state_of(slot, h), bytes, bar);
    } else {
      dt_mbar_arrive(bar);
    }
  };
  // the item after (e, h), and its position and slot (not looked at here, so that nothing waits for them)
  struct Where {
    int e, h, pos, slot;
  };
  auto look = [&](int e, int h) { return Where{e, h, e < nd ? ent.cached_lens[e] : 0, e < nd ? ent.slots[e] : -1}; };
  auto after = [&](const Where& w) { return w.h + 1 < H ? look(w.e, w.h + 1) : look(w.e + 1, 0); };
  auto gather = [&](const Where& x, bool first, RpdItem<T>& t) {
    const int e = x.e, h = x.h;
    t.same = !first && h % per != 0;
    t.ok = x.slot >= 0 && x.slot < rec.num_slots && x.pos >= 0 && e < ent.num_rows;
    if (!t.ok) {
      if (x.slot != -1 && tid == 0 && status) atomicOr(status, B200KV_S_BAD_POSITION);
      return;
    }
    t.row = e;
    t.head = h;
    t.slot = x.slot;
    t.fresh = x.pos == 0;
    t.at = x.pos % rec.taps;
    t.neg_a = rec.neg_a[h];
    t.skip = rec.skip ? rec.skip[h] : 0.f;
    if (norm.weight && tid < P) t.gate = ((const T*)norm.gate)[e * norm.gate_stride + h * P + tid];
    const T* xr = (const T*)in.x + e * in.x_stride;
    const T* sr = (const T*)in.step + e * in.step_stride;
    const T* ring = (const T*)rec.ring + (long long)x.slot * rec.taps * rec.channels;
    const int back = min(rec.taps - 1, x.pos);
    if (tid < D || tid < P4) {
      const int c = rec.channel_decay ? h * D + min(tid, D - 1) : h;
      t.step = sr[c];
      t.dt_bias = rec.dt_bias[c];
    }
    if (rec.correct) t.beta = ((const T*)in.beta)[e * in.beta_stride + h];
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      int k = tid + u * kRpdThreads;
      if (t.same) k = u == 0 && tid < P ? 2 * D + tid : -1;
      else if (k >= 2 * D + P) k = -1;
      t.k[u] = k;
      if (k < 0) continue;
      const int ch = channel(k, h);
      t.raw[u] = xr[ch];
      t.bias[u] = rec.conv_b ? rec.conv_b[ch] : 0.f;
      const float* w = rec.conv_w + (rec.taps - 1) * rec.channels + ch;
      const T* now = ring + t.at * rec.channels + ch;
#pragma unroll
      for (int j = 0; j < kRpdTaps; ++j) {
        const bool some = j <= back;
        t.w[u][j] = some ? w[-j * rec.channels] : 0.f;
        if (j > 0) t.past[u][j - 1] = some ? __ldcg(now + (t.at >= j ? -j : rec.taps - j) * rec.channels) : T(0);
      }
    }
  };
  const bool copier = tid == kRpdThreads - 32;  // in a warp that has no columns to add up
  if (copier)
    for (int i = 0; i < min(kRpdStages - 1, n); ++i) fetch(i);
  RpdItem<T> t;
  Where where = look(i0 / H, i0 % H);
  gather(where, true, t);
  where = after(where);
  const float norm_w = norm.weight && tid < P ? norm.weight[tid] : 0.f;
  const int c4 = tid % cg, r0 = tid / cg;
  const bool mine = r0 < rg;
  bool dead = false;
  for (int i = 0; i < n; ++i) {
    const bool ok = t.ok, fresh = t.fresh, same = t.same;
    const int row = t.row, h = t.head, slot = t.slot;
    const float skip = t.skip, gate = ld_elem(&t.gate);
    float beta = 0.f;
    if (ok) {
      float sq = 0.f, sk = 0.f;
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const int k = t.k[u];
        if (k < 0) continue;
        float v = fmaf(t.w[u][0], ld_elem(&t.raw[u]), t.bias[u]);
#pragma unroll
        for (int j = 1; j < kRpdTaps; ++j) v = fmaf(t.w[u][j], ld_elem(&t.past[u][j - 1]), v);
        v *= sigmoid_act<T>(v);
        // q and k inputs are kept by the first head of their group alone
        if (k >= 2 * D || h % per == 0) ((T*)rec.ring)[((long long)slot * rec.taps + t.at) * rec.channels + channel(k, h)] = t.raw[u];
        if (k < D) {
          qs[k] = v;
          sq = fmaf(v, v, sq);
        } else if (k < 2 * D) {
          ks[k - D] = v;
          sk = fmaf(v, v, sk);
        } else {
          vs[k - 2 * D] = v;
        }
      }
      if (tid < D || tid < P4) {
        const float step = softplus_f(ld_elem(&t.step) + t.dt_bias);
        beta = rec.correct ? sigmoid_f(ld_elem(&t.beta)) : step;
        if (tid < D) gs[tid] = expf(t.neg_a * step);
      }
      if (tid < P4 - P) vs[P + tid] = 0.f;
      if (!same) {
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        if ((tid & 31) == 0) {
          part[0][tid >> 5] = sq;
          part[1][tid >> 5] = sk;
        }
      }
    }
    __syncthreads();
    if (i + 1 < n) {
      gather(where, !ok, t);
      where = after(where);
    }
    if (copier && i + kRpdStages - 1 < n) {  // into the stage of the item before, once its copy out has been read
      asm volatile("cp.async.bulk.wait_group.read 0;\n" ::: "memory");
      fetch(i + kRpdStages - 1);
    }
    float qk = 0.f;
    if (ok && !same) {
      if (tid < D) qk = qs[tid] * ks[tid];
      qk = warp_sum(qk);
      if ((tid & 31) == 0) part[2][tid >> 5] = qk;
    }
    if (!dt_mbar_wait(dt_smem(bars + i % kRpdStages), (i / kRpdStages) & 1)) dead = true;
    float* st = stage(i);
    ulonglong2 S[kRows];
    if (ok && !dead && mine) {
      ulonglong2 ak = make_ulonglong2(0ull, 0ull), aq = ak;
#pragma unroll
      for (int j = 0; j < kRows; ++j) {
        const int d = r0 + j * rg;
        if (d >= D) break;
        ulonglong2 s = make_ulonglong2(0ull, 0ull);
        if (!fresh) s = *reinterpret_cast<const ulonglong2*>(st + d * P4 + 4 * c4);
        const rpd_pair g = rpd_both(gs[d]), k = rpd_both(ks[d]), q = rpd_both(qs[d]);
        s.x = rpd_mul(s.x, g);
        s.y = rpd_mul(s.y, g);
        ak.x = rpd_fma(s.x, k, ak.x);
        ak.y = rpd_fma(s.y, k, ak.y);
        aq.x = rpd_fma(s.x, q, aq.x);
        aq.y = rpd_fma(s.y, q, aq.y);
        S[j] = s;
      }
      *reinterpret_cast<ulonglong2*>(red + r0 * 4 * cg + 4 * c4) = ak;
      *reinterpret_cast<ulonglong2*>(red + (rg + r0) * 4 * cg + 4 * c4) = aq;
    }
    __syncthreads();
    float ss = 0.f;
    if (ok && tid < P4) {  // one thread per column
      float sq = 0.f, sk = 0.f, dot = 0.f, rk = 0.f, rq = 0.f;
#pragma unroll
      for (int w = 0; w < kRpdThreads / 32; ++w) {
        sq += part[0][w];
        sk += part[1][w];
        dot += part[2][w];
      }
      const float fq = rec.q_scale * (rec.unit_norm ? 1.0f / sqrtf(sq + rec.unit_eps) : 1.f);
      const float fk = rec.unit_norm ? 1.0f / sqrtf(sk + rec.unit_eps) : 1.f;
#pragma unroll 8
      for (int r = 0; r < rg; ++r) {
        rk += red[r * 4 * cg + tid];
        rq += red[(rg + r) * 4 * cg + tid];
      }
      const float v = vs[tid], u = rec.correct ? beta * fmaf(-fk, rk, v) : beta * v;
      us[tid] = fk * u;
      const float o = fmaf(skip, v, fmaf(dot * fq * fk, u, fq * rq));
      os[tid] = o;
      if (!norm.weight) {
        if (tid < P && !dead) ((float*)out)[((long long)row * H + h) * P + tid] = o;
      } else {
        ss = o * o;
      }
    }
    if (norm.weight) ss = warp_sum(ss);
    __syncthreads();
    if (norm.weight && (tid & 31) == 0) part[3][tid >> 5] = ss;
    if (ok && !dead && mine) {
      const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(us + 4 * c4);
#pragma unroll
      for (int j = 0; j < kRows; ++j) {
        const int d = r0 + j * rg;
        if (d >= D) break;
        const rpd_pair k = rpd_both(ks[d]);
        *reinterpret_cast<ulonglong2*>(st + d * P4 + 4 * c4) = make_ulonglong2(rpd_fma(k, u.x, S[j].x), rpd_fma(k, u.y, S[j].y));
      }
    }
    asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");  // the new state, for the copy out
    const bool stop = __syncthreads_or(dead);
    if (stop) {
      if (copier) {
        if (status) atomicOr(status, B200KV_S_TIMEOUT);
        for (int j = i; j < min(i + kRpdStages, n); ++j) dt_mbar_wait(dt_smem(bars + j % kRpdStages), (j / kRpdStages) & 1);
        asm volatile("cp.async.bulk.wait_group 0;\n" ::: "memory");
      }
      __syncthreads();
      return;
    }
    if (copier && ok) rpd_store(state_of(slot, h), dt_smem(st), bytes);
    if (norm.weight && ok) {
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < kRpdThreads / 32; ++w) sum += part[3][w];
      if (tid < P) {
        const float inv = 1.0f / sqrtf(sum / (float)P + norm.eps);
        st_elem((T*)out + row * norm.out_stride + h * P + tid, os[tid] * inv * norm_w * sigmoid_act<T>(gate));
      }  // os and part[3] are written again behind two barriers of the next item
    }
  }
  if (copier) asm volatile("cp.async.bulk.wait_group 0;\n" ::: "memory");
}

struct RpdShape {
  int threads, cg, rg, rows, blocks_per_sm;
  size_t smem;
};
static bool rpd_shape(const b200dec_recurrence& r, RpdShape* s) {
  const int quads = rec_round4(r.vdim) / 4;
  const size_t floats = ((size_t)r.dim * 4 * quads + 31) / 32 * 32;
  s->threads = floats * 4 > 16 * 1024 || 2 * r.dim + r.vdim > 256 || quads > 32 ? 256 : 128;  // small states: more and smaller blocks
  if (r.taps > kRpdTaps || quads > 64 || 2 * r.dim + r.vdim > 2 * s->threads) return false;
  s->cg = quads;
  s->rg = s->threads / quads;
  s->rows = (r.dim + s->rg - 1) / s->rg;
  s->smem = (kRpdStages * floats + 3 * rec_round4(r.dim) + 3 * 4 * quads + (size_t)8 * s->rg * quads) * 4;
  if (s->rows > (s->threads == 256 ? 16 : 8) || s->smem > 225 * 1024) return false;
  const int fit = (int)(227 * 1024 / (s->smem + 1024 + 512)), regs = s->rows > 8 ? 1 : 512 / s->threads;
  s->blocks_per_sm = fit < regs ? fit : regs;
  return true;
}

template <typename T, int kRows, int kThreads>
static int rpd_launch(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const b200dec_entries& ent, const RecNorm& norm, void* out,
                      const RpdShape& sh, int sm_count, int32_t* status, cudaStream_t s) {
  auto* kernel = recurrence_step_kernel<T, kRows, kThreads>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sh.smem) != cudaSuccess) return B200KV_E_LAUNCH;
  const long long items = (long long)ent.num_entries * rec.heads, most = (long long)sm_count * sh.blocks_per_sm;
  return launch_result(launch_chained(kernel, dim3((unsigned)(items < most ? items : most)), dim3(kThreads), sh.smem, s, rec, in, ent, norm, out,
                                      sh.cg, sh.rg, status));
}

template <typename T>
static int rpd_run(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const b200dec_entries& ent, const RecNorm& norm, void* out,
                   const RpdShape& sh, int sm_count, int32_t* status, cudaStream_t s) {
  if (sh.threads == 128 && sh.rows <= 4) return rpd_launch<T, 4, 128>(rec, in, ent, norm, out, sh, sm_count, status, s);
  if (sh.threads == 128) return rpd_launch<T, 8, 128>(rec, in, ent, norm, out, sh, sm_count, status, s);
  if (sh.rows <= 4) return rpd_launch<T, 4, 256>(rec, in, ent, norm, out, sh, sm_count, status, s);
  if (sh.rows <= 8) return rpd_launch<T, 8, 256>(rec, in, ent, norm, out, sh, sm_count, status, s);
  return rpd_launch<T, 16, 256>(rec, in, ent, norm, out, sh, sm_count, status, s);
}

int recurrence_decode_any(const b200dec_recurrence& rec, const b200dec_recurrence_in& in, const b200dec_entries& ent, const RecNorm& norm,
                          void* out, int32_t* status, cudaStream_t s);  // recurrence.cu

}  // namespace b200kv

using namespace b200kv;

extern "C" int b200dec_recurrence_decode(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const b200dec_entries* ent,
                                         const float* norm_w, float eps, const void* gate, int64_t gate_stride, void* out,
                                         int64_t out_stride, int32_t variant, int32_t sm_count, int32_t* status, void* stream) {
  const int rc = check_recurrence(rec, in, ent);
  if (rc != B200KV_OK) return rc;
  if (ent->num_entries == 0) return B200KV_OK;
  if (!out || (norm_w && !gate)) return B200KV_E_NULL;
  if (sm_count < 1 || (long long)ent->num_entries * rec->heads > 0x3FFFFFFFll || (long long)rec->taps * rec->channels > 0x7FFFFFFFll)
    return B200KV_E_RANGE;
  const RecNorm norm{norm_w, gate, gate_stride, out_stride, eps};
  cudaStream_t s = (cudaStream_t)stream;
  RpdShape sh;
  if (variant != 0 || !rpd_shape(*rec, &sh)) return recurrence_decode_any(*rec, *in, *ent, norm, out, status, s);
  return rec->elem == 2 ? rpd_run<uint16_t>(*rec, *in, *ent, norm, out, sh, sm_count, status, s)
                        : rpd_run<float>(*rec, *in, *ent, norm, out, sh, sm_count, status, s);
}
