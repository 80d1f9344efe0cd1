// Decode attention over the paged bf16 cache (key and value sizes up to 128, any number of query heads per kv head).
// HBM-bound: every key and value is read once per group of query heads.
//
// Work: the unit is a block of 64 keys of one (entry, kv head, group of up to 16 query heads).  All units of the batch
// lie end to end in (entry, head, block) order and are cut into equal ranges, one per CTA of a persistent grid (two
// CTAs per SM), from cached_lens on the device: the grid depends on shapes only.
// One CTA: a producer warp fetches blocks by page with tensor-map copies into a ring of stages; four consumer warps own
// 16 of a block's 64 keys each and run S = Q K^T and O += P V as bf16 mma.m16n8k16 with 32-bit scores, softmax state and
// sums (query heads are the 16 rows of the product).  When the CTA's part of an (entry, head) ends, the four warps are
// added up in shared memory; a part that is the whole of it is written out, otherwise it goes to the workspace and the
// CTA that delivers the last part adds them (arrival counters return to zero).
// With a sliding window only the blocks that hold a visible key are units; a sink joins the softmax sum when an (entry,
// head) is complete, and the output gate multiplies there.
// Every wait is bounded: when one runs out the CTA goes on without waiting, writes nothing and sets B200KV_S_TIMEOUT.
#include "dec_tma.cuh"

namespace b200kv {

constexpr int kPdKeys = 64;      // keys per block
constexpr int kPdWarps = 4;      // consumer warps
constexpr int kPdThreads = 32 * (kPdWarps + 1);
constexpr int kPdRows = 16;      // query heads per unit
constexpr int kPdCtasPerSm = 2;
constexpr int kPdMinBlocks = 4;  // smallest share of a CTA
constexpr uint32_t kPdBlockBytes = kPdKeys * 128;  // 64 rows x 64 channels
constexpr int kPdMaxB = 4096;

__host__ __device__ constexpr int pd_stages(int kb, int vb) { return kb + vb == 4 ? 3 : (kb + vb == 3 ? 4 : 6); }

__device__ __forceinline__ void pd_ldsm(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void pd_ldsm_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void pd_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float pd_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t pd_pack(float lo, float hi) {
  uint32_t r;
  asm("cvt.rn.bf16x2.f32 %0, %1, %2;\n" : "=r"(r) : "f"(hi), "f"(lo));
  return r;
}
__device__ __forceinline__ void pd_sync() { asm volatile("bar.sync 1, %0;\n" ::"n"(32 * kPdWarps) : "memory"); }
__device__ __forceinline__ int pd_arrive(int* addr) {  // release my stores, acquire the others'
  int old;
  asm volatile("atom.add.acq_rel.gpu.global.s32 %0, [%1], 1;" : "=r"(old) : "l"(addr) : "memory");
  return old;
}

// First block of 64 keys that a query at position len (its own key the last) sees, and the number of such blocks.
__device__ __forceinline__ int pd_first(int len, int window) { return window > 0 ? max(0, len - window + 1) / kPdKeys : 0; }
__device__ __forceinline__ int pd_blocks(int len, int window) {
  len = max(len, 0);
  return (len + kPdKeys) / kPdKeys - pd_first(len, window);
}

// Position in the flattened (entry, head unit, block) list.
struct PdCursor {
  int b, hu, blk, nb, n;  // n: keys of the entry
  __device__ __forceinline__ void entry(const int* pre, const int32_t* lens, int bb) {
    b = bb;
    nb = pre[bb + 1] - pre[bb];
    n = nb > 0 ? lens[bb] + 1 : 0;
  }
  __device__ __forceinline__ void seek(const int* pre, const int32_t* lens, int B, int HU, int u) {
    int lo = 0, hi = B;  // largest b with HU * pre[b] <= u
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (HU * pre[mid] <= u) lo = mid; else hi = mid;
    }
    entry(pre, lens, lo);
    const int r = u - HU * pre[lo];
    hu = r / nb;
    blk = r - hu * nb;
  }
  __device__ __forceinline__ void next_unit(const int* pre, const int32_t* lens, int HU) {  // only while one exists
    blk = 0;
    if (++hu < HU) return;
    hu = 0;
    int bb = b + 1;
    while (pre[bb + 1] == pre[bb]) ++bb;
    entry(pre, lens, bb);
  }
};

template <int KB, int VB, bool kWide>
__global__ void __launch_bounds__(kPdThreads, kPdCtasPerSm)
paged_decode_kernel(const uint16_t* __restrict__ q, DecCache c, const int32_t* __restrict__ cached_lens,
                    const int32_t* __restrict__ num_decoding, int B, int heads, int groups, float scale_log2, DecAttnOpt opt,
                    uint16_t* __restrict__ out, int zero_idle, int* __restrict__ counters, float* __restrict__ parts, int box_rows, int32_t* status,
                    const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v) {
  extern __shared__ uint8_t pd_raw[];
  constexpr int kStages = pd_stages(KB, VB);
  constexpr uint32_t kStageBytes = (KB + VB) * kPdBlockBytes;
  constexpr int kTiles = 8 * VB;                        // 8-channel tiles of O
  constexpr int kPart = kPdRows * (64 * VB + 2);        // floats of one part: O rows, then m and l
  __shared__ float ml[kPdWarps][kPdRows][2];
  __shared__ float obuf[kTiles * 4 * 32];
  __shared__ __align__(8) uint64_t bars[2 * kStages];
  __shared__ int sums[kPdThreads];
  __shared__ int flag_last, flag_dead;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t stage0 = (dt_smem(pd_raw) + 1023u) & ~1023u;
  int* pre = reinterpret_cast<int*>(pd_raw + (stage0 - dt_smem(pd_raw)) + kStages * kStageBytes);  // [B + 1] blocks before entry b
  const uint32_t bar0 = dt_smem(bars);
  auto full = [&](int s) { return bar0 + 8 * s; };
  auto empty = [&](int s) { return bar0 + 8 * (kStages + s); };
  if ((blockIdx.x) == 0) pdl_wait();  // a grid in which no CTA waited could complete before its predecessor
  const int nd = max(0, min(*num_decoding, B));
  {
    const int chunk = (B + kPdThreads - 1) / kPdThreads, lo = min(tid * chunk, B), hi = min(lo + chunk, B);
    int sum = 0;
    for (int b = lo; b < hi; ++b) sum += b < nd ? pd_blocks(cached_lens[b], opt.window) : 0;
    sums[tid] = sum;
    if (tid == 0) {
      for (int s = 0; s < kStages; ++s) {
        dt_mbar_init(full(s), 1);
        dt_mbar_init(empty(s), kPdWarps);
      }
      flag_dead = 0;
      asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
    }
    __syncthreads();
    if (tid < 32) {
      int carry = 0;
      for (int base = 0; base < kPdThreads; base += 32) {
        const int v = sums[base + tid];
        int incl = v;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const int y = __shfl_up_sync(0xffffffffu, incl, o);
          if (tid >= o) incl += y;
        }
        sums[base + tid] = carry + incl - v;
        carry += __shfl_sync(0xffffffffu, incl, 31);
      }
      if (tid == 0) pre[B] = carry;
    }
    __syncthreads();
    int run = sums[tid];
    for (int b = lo; b < hi; ++b) {
      pre[b] = run;
      run += b < nd ? pd_blocks(cached_lens[b], opt.window) : 0;
    }
    __syncthreads();
  }
  pdl_wait();
  if (zero_idle) {
    const int row = heads * c.v_dim;
    for (int b = nd + blockIdx.x; b < B; b += gridDim.x)
      for (int i = tid; i < row; i += kPdThreads) out[b * opt.out_stride + i] = 0;
  }
  const int HU = c.heads * groups, total = HU * pre[B];
  const int per = max((total + (int)gridDim.x - 1) / (int)gridDim.x, kPdMinBlocks);
  const long long u0l = (long long)blockIdx.x * per;
  if (u0l >= total) { pdl_trigger(); return; }
  const int u0 = (int)u0l, u1 = min(u0 + per, total);
  const int G = heads / c.heads;
  PdCursor cur;
  cur.seek(pre, cached_lens, B, HU, u0);

  if (warp == kPdWarps) {  // ---- producer
    if (lane == 0) {
      bool live = true;
      int i = 0;
      for (int u = u0; u < u1 && live; ++u, ++i) {
        const int s = i % kStages;
        if (i >= kStages && !dt_mbar_wait(empty(s), (i / kStages - 1) & 1)) { live = false; break; }
        const int key0 = (pd_first(cur.n - 1, opt.window) + cur.blk) * kPdKeys;
        const int nbox = (min(kPdKeys, cur.n - key0) + box_rows - 1) / box_rows;
        const int hk = cur.hu / groups;
        dt_expect_tx(full(s), (uint32_t)nbox * box_rows * 128 * (KB + VB));
        const uint32_t dst = stage0 + s * kStageBytes;
        for (int x = 0; x < nbox; ++x) {
          const int pos = key0 + x * box_rows;
          int page = dec_page(c, cur.b, pos, status);
          if (page < 0) page = 0;  // reported; the copy stays inside the cache
          const int prow = pos % c.P, ph = page * c.heads + hk;
#pragma unroll
          for (int k = 0; k < KB; ++k) dt_tma_3d(dst + k * kPdBlockBytes + x * box_rows * 128, &tm_k, 64 * k, prow, ph, full(s));
#pragma unroll
          for (int k = 0; k < VB; ++k) dt_tma_3d(dst + (KB + k) * kPdBlockBytes + x * box_rows * 128, &tm_v, 64 * k, prow, ph, full(s));
        }
        if (++cur.blk == cur.nb && u + 1 < u1) cur.next_unit(pre, cached_lens, HU);
      }
      pdl_trigger();
      if (!live) {  // the copies in flight land before the CTA may end
        if (status) atomicOr(status, B200KV_S_TIMEOUT);
        for (int k = max(0, i - kStages); k < i; ++k) dt_mbar_wait(full(k % kStages), (k / kStages) & 1);
      }
    }
    return;
  }

  // ---- consumers
  const int g = lane >> 2, t = lane & 3, mi = lane >> 3, mr = lane & 7;
  const int k_key = warp * 16 + (mi >> 1) * 8 + mr, k_sel = mi & 1;  // ldmatrix lane addressing: K tile (keys x channels)
  const int v_key = warp * 16 + (mi & 1) * 8 + mr, v_sel = mi >> 1;  // V tile, transposed on the way
  bool dead = false;
  int i = 0;
  for (int u = u0; u < u1;) {
    // one segment: this CTA's part of (entry, head unit)
    const int hk = cur.hu / groups, gq = cur.hu - hk * groups;
    const int head0 = hk * G + gq * kPdRows, nh = min(kPdRows, G - gq * kPdRows);
    const int ublk = cur.blk, nblk = min(cur.nb - cur.blk, u1 - u);
    const bool whole = ublk == 0 && nblk == cur.nb;
    const int lo = opt.window > 0 ? max(0, cur.n - opt.window) : 0, blk0 = pd_first(cur.n - 1, opt.window) + ublk;
    uint32_t qa[4 * KB][4];
    {
      const uint16_t* r0 = q + ((long long)cur.b * heads + head0 + g) * c.k_row;
      const uint16_t* r1 = r0 + 8 * c.k_row;
#pragma unroll
      for (int s = 0; s < 4 * KB; ++s)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int ch = 16 * s + 8 * e + 2 * t;
          qa[s][2 * e] = (g < nh && ch < c.k_row) ? *reinterpret_cast<const uint32_t*>(r0 + ch) : 0u;
          qa[s][2 * e + 1] = (kWide && g + 8 < nh && ch < c.k_row) ? *reinterpret_cast<const uint32_t*>(r1 + ch) : 0u;
        }
    }
    float o[kTiles][4];
#pragma unroll
    for (int j = 0; j < kTiles; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    for (int k = 0; k < nblk; ++k, ++i) {
      const int s = i % kStages;
      if (!dead && !dt_mbar_wait(full(s), (i / kStages) & 1)) dead = true;
      const int nvalid = cur.n - (blk0 + k) * kPdKeys - warp * 16;  // keys of this warp's tile
      const int nskip = lo - (blk0 + k) * kPdKeys - warp * 16;      // ... and those in front of the window
      if (nvalid > 0 && nskip < 16 && !dead) {
        const uint32_t sk = stage0 + s * kStageBytes, sv = sk + KB * kPdBlockBytes;
        float sc[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < 4 * KB; ++ks) {
          const int chunk = 2 * ks + k_sel;
          uint32_t b[4];
          pd_ldsm(b, sk + (chunk >> 3) * kPdBlockBytes + k_key * 128 + (((chunk & 7) ^ (k_key & 7)) << 4));
          pd_mma(sc[0], qa[ks], b[0], b[1]);
          pd_mma(sc[1], qa[ks], b[2], b[3]);
        }
        // sc[j][0..1]: head g, keys 8j + 2t, +1;  sc[j][2..3]: head g + 8
        float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int key = 8 * j + 2 * t + e;
            const bool in = key < nvalid && key >= nskip;
            sc[j][e] = in ? sc[j][e] * scale_log2 : -INFINITY;
            mx0 = fmaxf(mx0, sc[j][e]);
            if (kWide) {
              sc[j][2 + e] = in ? sc[j][2 + e] * scale_log2 : -INFINITY;
              mx1 = fmaxf(mx1, sc[j][2 + e]);
            }
          }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        if (kWide) {
          mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
          mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        }
        const bool grow = mx0 > m0 || (kWide && mx1 > m1);
        if (__any_sync(0xffffffffu, grow)) {
          const float n0 = fmaxf(m0, mx0), n1 = fmaxf(m1, mx1);
          const float a0 = m0 == -INFINITY ? 0.f : pd_exp2(m0 - n0), a1 = m1 == -INFINITY ? 0.f : pd_exp2(m1 - n1);
          m0 = n0; m1 = n1;
          l0 *= a0; l1 *= a1;
#pragma unroll
          for (int j = 0; j < kTiles; ++j) {
            o[j][0] *= a0; o[j][1] *= a0;
            if (kWide) { o[j][2] *= a1; o[j][3] *= a1; }
          }
        }
        const float b0 = m0 == -INFINITY ? 0.f : m0, b1 = m1 == -INFINITY ? 0.f : m1;
        uint32_t pa[4];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const float p0 = pd_exp2(sc[j][0] - b0), p1 = pd_exp2(sc[j][1] - b0);
          l0 += p0 + p1;
          pa[2 * j] = pd_pack(p0, p1);
          if (kWide) {
            const float p2 = pd_exp2(sc[j][2] - b1), p3 = pd_exp2(sc[j][3] - b1);
            l1 += p2 + p3;
            pa[2 * j + 1] = pd_pack(p2, p3);
          } else {
            pa[2 * j + 1] = 0u;
          }
        }
        // rows behind the sequence may hold anything, also what is not a number: their values are cleared
        const uint32_t keep0 = (2 * t < nvalid ? 0xFFFFu : 0u) | (2 * t + 1 < nvalid ? 0xFFFF0000u : 0u);
        const uint32_t keep1 = (2 * t + 8 < nvalid ? 0xFFFFu : 0u) | (2 * t + 9 < nvalid ? 0xFFFF0000u : 0u);
#pragma unroll
        for (int j = 0; j < kTiles / 2; ++j) {
          const int chunk = 2 * j + v_sel;
          uint32_t b[4];
          pd_ldsm_t(b, sv + (chunk >> 3) * kPdBlockBytes + v_key * 128 + (((chunk & 7) ^ (v_key & 7)) << 4));
          if (nvalid < 16) { b[0] &= keep0; b[1] &= keep1; b[2] &= keep0; b[3] &= keep1; }
          pd_mma(o[2 * j], pa, b[0], b[1]);
          pd_mma(o[2 * j + 1], pa, b[2], b[3]);
        }
      }
      __syncwarp();
      if (lane == 0) dt_mbar_arrive(empty(s));
    }
    u += nblk;

    // ---- the four warps' parts become one, in warp 0
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    if (t == 0) {
      ml[warp][g][0] = m0; ml[warp][g][1] = l0;
      ml[warp][g + 8][0] = m1; ml[warp][g + 8][1] = l1;
    }
    if (dead) flag_dead = 1;
    pd_sync();
    float M0 = -INFINITY, M1 = -INFINITY, L0 = 0.f, L1 = 0.f;
#pragma unroll
    for (int w = 0; w < kPdWarps; ++w) {
      M0 = fmaxf(M0, ml[w][g][0]);
      M1 = fmaxf(M1, ml[w][g + 8][0]);
    }
    float sink0 = -INFINITY, sink1 = -INFINITY;
    if (whole && opt.sink) {
      if (g < nh) sink0 = opt.sink[head0 + g] * 1.4426950408889634f;
      if (kWide && g + 8 < nh) sink1 = opt.sink[head0 + g + 8] * 1.4426950408889634f;
      M0 = fmaxf(M0, sink0);
      M1 = fmaxf(M1, sink1);
    }
    const float B0 = M0 == -INFINITY ? 0.f : M0, B1 = M1 == -INFINITY ? 0.f : M1;
    if (whole && opt.sink) {
      L0 = pd_exp2(sink0 - B0);
      L1 = pd_exp2(sink1 - B1);
    }
#pragma unroll
    for (int w = 0; w < kPdWarps; ++w) {
      L0 += ml[w][g][1] * pd_exp2(ml[w][g][0] - B0);
      L1 += ml[w][g + 8][1] * pd_exp2(ml[w][g + 8][0] - B1);
    }
    const float f0 = pd_exp2(m0 - B0), f1 = pd_exp2(m1 - B1);
#pragma unroll
    for (int j = 0; j < kTiles; ++j) {
      o[j][0] *= f0; o[j][1] *= f0;
      o[j][2] *= f1; o[j][3] *= f1;
    }
    for (int w = kPdWarps - 1; w >= 0; --w) {
      if (warp == w) {
        if (w < kPdWarps - 1) {
#pragma unroll
          for (int j = 0; j < kTiles; ++j)
#pragma unroll
            for (int e = 0; e < (kWide ? 4 : 2); ++e) o[j][e] += obuf[(4 * j + e) * 32 + lane];
        }
        if (w > 0) {
#pragma unroll
          for (int j = 0; j < kTiles; ++j)
#pragma unroll
            for (int e = 0; e < (kWide ? 4 : 2); ++e) obuf[(4 * j + e) * 32 + lane] = o[j][e];
        }
      }
      if (w > 0) pd_sync();
    }
    const bool lost = *(volatile int*)&flag_dead != 0;
    if (lost && status && tid == 0) atomicOr(status, B200KV_S_TIMEOUT);
    const long long orow = cur.b * opt.out_stride + head0 * c.v_dim;
    if (whole) {
      if (warp == 0 && !lost) {
        const float i0 = (L0 > 0.f ? 1.f / L0 : 0.f) * (g < nh ? opt.factor<uint16_t>(cur.b, head0 + g) : 0.f);
        const float i1 = (L1 > 0.f ? 1.f / L1 : 0.f) * (kWide && g + 8 < nh ? opt.factor<uint16_t>(cur.b, head0 + g + 8) : 0.f);
        const bool pairs = c.v_dim % 2 == 0 && opt.out_stride % 2 == 0;
#pragma unroll
        for (int j = 0; j < kTiles; ++j)
#pragma unroll
          for (int half = 0; half < (kWide ? 2 : 1); ++half) {
            const int row = g + 8 * half, ch = 8 * j + 2 * t;
            const float y0 = o[j][2 * half] * (half ? i1 : i0), y1 = o[j][2 * half + 1] * (half ? i1 : i0);
            uint16_t* dst = out + orow + (long long)row * c.v_dim + ch;
            if (row < nh && ch < c.v_dim) {
              if (pairs) {
                *reinterpret_cast<uint32_t*>(dst) = pd_pack(y0, y1);
              } else {
                st_elem(dst, y0);
                if (ch + 1 < c.v_dim) st_elem(dst + 1, y1);
              }
            }
          }
      }
    } else if (!lost) {
      // unit range [a, z) of this (entry, head unit) in the flat list, and the CTAs that share it
      const int a = u - nblk - ublk, z = a + cur.nb;
      const int c_lo = a / per, c_hi = (z - 1) / per;
      const int mine = blockIdx.x, slot = a <= mine * per ? 0 : 1;
      if (warp == 0) {
        float* p = parts + (long long)(2 * mine + slot) * kPart;
#pragma unroll
        for (int j = 0; j < kTiles; ++j)
#pragma unroll
          for (int half = 0; half < (kWide ? 2 : 1); ++half)
            *reinterpret_cast<float2*>(p + (g + 8 * half) * (64 * VB) + 8 * j + 2 * t) = make_float2(o[j][2 * half], o[j][2 * half + 1]);
        if (t == 0) {
          p[kPdRows * 64 * VB + g] = M0; p[kPdRows * 64 * VB + kPdRows + g] = L0;
          p[kPdRows * 64 * VB + g + 8] = M1; p[kPdRows * 64 * VB + kPdRows + g + 8] = L1;
        }
        __threadfence();
        __syncwarp();
        if (lane == 0) flag_last = pd_arrive(counters + cur.b * HU + cur.hu) == c_hi - c_lo;
      }
      pd_sync();
      if (flag_last) {
        __threadfence();
        for (int x = tid; x < nh * 64 * VB; x += 32 * kPdWarps) {
          const int row = x / (64 * VB), ch = x - row * (64 * VB);
          if (ch >= c.v_dim) continue;
          const float sink = opt.sink ? opt.sink[head0 + row] * 1.4426950408889634f : -INFINITY;
          float M = sink;
          for (int cc = c_lo; cc <= c_hi; ++cc) {
            const float* p = parts + (long long)(2 * cc + (a <= cc * per ? 0 : 1)) * kPart;
            M = fmaxf(M, __ldcg(p + kPdRows * 64 * VB + row));
          }
          const float base = M == -INFINITY ? 0.f : M;
          float L = opt.sink ? pd_exp2(sink - base) : 0.f, acc = 0.f;
          for (int cc = c_lo; cc <= c_hi; ++cc) {
            const float* p = parts + (long long)(2 * cc + (a <= cc * per ? 0 : 1)) * kPart;
            const float f = pd_exp2(__ldcg(p + kPdRows * 64 * VB + row) - base);
            L = fmaf(f, __ldcg(p + kPdRows * 64 * VB + kPdRows + row), L);
            acc = fmaf(f, __ldcg(p + row * (64 * VB) + ch), acc);
          }
          st_elem(out + orow + (long long)row * c.v_dim + ch, L > 0.f ? acc / L * opt.factor<uint16_t>(cur.b, head0 + row) : 0.f);
        }
        if (tid == 0) counters[cur.b * HU + cur.hu] = 0;
      }
    }
    pd_sync();  // ml, obuf and the flag are free again
    cur.blk += nblk;
    if (u < u1) cur.next_unit(pre, cached_lens, HU);
  }
}

template <int KB, int VB, bool kWide>
static int pd_launch(const void* q, const DecCache& c, const int32_t* cached_lens, const int32_t* num_decoding, int B, int heads, int groups,
                     float scale_log2, const DecAttnOpt& opt, void* out, int zero_idle, int* counters, float* parts, int grid, int box_rows, int32_t* status,
                     const CUtensorMap& tm_k, const CUtensorMap& tm_v, cudaStream_t stream) {
  const size_t smem = (size_t)pd_stages(KB, VB) * (KB + VB) * kPdBlockBytes + 1024 + (size_t)(B + 1) * 4;
  if (cudaFuncSetAttribute(paged_decode_kernel<KB, VB, kWide>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return B200KV_E_LAUNCH;
  return launch_result(launch_chained(paged_decode_kernel<KB, VB, kWide>, dim3(grid), dim3(kPdThreads), smem, stream, (const uint16_t*)q, c,
                                      cached_lens, num_decoding, B, heads, groups, scale_log2, opt, (uint16_t*)out, zero_idle, counters, parts,
                                      box_rows, status, tm_k, tm_v));
}

}  // namespace b200kv

using namespace b200kv;

static size_t pd_counter_bytes(int B, int heads) { return ((size_t)B * heads * 4 + 255) / 256 * 256; }

extern "C" size_t b200dec_decode_attn_workspace(int32_t B, int32_t heads, int32_t kv_heads, int32_t v_dim, int32_t sm_count) {
  if (B < 1 || heads < 1 || kv_heads < 1 || v_dim < 1 || sm_count < 1) return 0;
  const int vb = v_dim <= 64 ? 1 : 2;
  // counters per (entry, head unit): there are never more units than query heads
  return pd_counter_bytes(B, heads) + (size_t)sm_count * kPdCtasPerSm * 2 * kPdRows * (64 * vb + 2) * 4;
}

extern "C" int b200dec_decode_attn_opt(const void* q, const b200dec_cache* cache, const b200kv_table* table, const int32_t* cached_lens,
                                       const int32_t* num_decoding, int32_t B, int32_t heads, float scale,
                                       const b200dec_attn_options* options, void* out, int32_t zero_idle, void* workspace,
                                       size_t workspace_bytes, int32_t sm_count, int32_t* status, void* stream) {
  if (B == 0) return B200KV_OK;
  if (!q || !cached_lens || !num_decoding || !out || !workspace) return B200KV_E_NULL;
  const int rc = check_dec_cache(cache, table);
  if (rc != B200KV_OK) return rc;
  if (cache->elem != 2 || cache->k_dim > 128 || cache->v_dim > 128 || cache->page_size % 16 || heads < 1 || heads % cache->kv_heads)
    return B200KV_E_SHAPE;
  if (B < 0 || B > kPdMaxB || sm_count < 1 || (long long)cache->num_pages * cache->kv_heads > 0x7FFFFFFFll ||
      (long long)B * heads * table->max_pages * ((cache->page_size + kPdKeys - 1) / kPdKeys) > 0x3FFFFFFFll)
    return B200KV_E_RANGE;
  DecAttnOpt opt;
  const int bad = dec_attn_opt(options, heads, cache->v_dim, &opt);
  if (bad != B200KV_OK) return bad;
  if (!aligned(q, 16) || !aligned(out, 4) || !aligned(workspace, 256)) return B200KV_E_ALIGN;
  if (workspace_bytes < b200dec_decode_attn_workspace(B, heads, cache->kv_heads, cache->v_dim, sm_count)) return B200KV_E_WORKSPACE;
  const DecCache c = dec_view(cache, table);
  const int G = heads / c.heads, groups = (G + kPdRows - 1) / kPdRows, box = dec_box_rows(c.P);
  CUtensorMap tm_k, tm_v;
  const long long ph = (long long)c.num_pages * c.heads;
  if (!dt_cache_map(&tm_k, c.k, c.k_dim, c.k_row, c.P, ph, box) || !dt_cache_map(&tm_v, c.v, c.v_dim, c.v_row, c.P, ph, box))
    return B200KV_E_LAUNCH;
  int* counters = (int*)workspace;
  float* parts = (float*)((uint8_t*)workspace + pd_counter_bytes(B, heads));
  // no more CTAs than the largest batch the table can address has shares of the smallest size
  long long entry_blocks = ((long long)c.max_pages * c.P + kPdKeys - 1) / kPdKeys;
  if (opt.window > 0 && entry_blocks > opt.window / kPdKeys + 2) entry_blocks = opt.window / kPdKeys + 2;
  const long long units = (long long)B * c.heads * groups * entry_blocks;
  const long long want = (units + kPdMinBlocks - 1) / kPdMinBlocks;
  const int grid = (int)(want < (long long)sm_count * kPdCtasPerSm ? want : (long long)sm_count * kPdCtasPerSm);
  const float sl = scale * 1.4426950408889634f;
  const int kb = c.k_dim > 64, vb = c.v_dim > 64, wide = G > 8;
  cudaStream_t s = (cudaStream_t)stream;
#define PD_CASE(KB, VB, W)                                                                                                        \
  if (kb == KB - 1 && vb == VB - 1 && wide == W)                                                                                  \
    return pd_launch<KB, VB, W>(q, c, cached_lens, num_decoding, B, heads, groups, sl, opt, out, zero_idle, counters, parts, grid, box, \
                                status, tm_k, tm_v, s);
  PD_CASE(1, 1, false) PD_CASE(1, 1, true) PD_CASE(1, 2, false) PD_CASE(1, 2, true)
  PD_CASE(2, 1, false) PD_CASE(2, 1, true) PD_CASE(2, 2, false) PD_CASE(2, 2, true)
#undef PD_CASE
  return B200KV_E_SHAPE;
}

extern "C" int b200dec_decode_attn(const void* q, const b200dec_cache* cache, const b200kv_table* table, const int32_t* cached_lens,
                                   const int32_t* num_decoding, int32_t B, int32_t heads, float scale, void* out, int32_t zero_idle,
                                   void* workspace, size_t workspace_bytes, int32_t sm_count, int32_t* status, void* stream) {
  return b200dec_decode_attn_opt(q, cache, table, cached_lens, num_decoding, B, heads, scale, nullptr, out, zero_idle, workspace,
                                 workspace_bytes, sm_count, status, stream);
}
