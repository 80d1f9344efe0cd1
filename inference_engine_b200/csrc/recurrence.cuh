// Device views and element-wise parts shared by the recurrent-layer kernels.
#pragma once
#include "dec_common.cuh"

namespace b200kv {

struct RecEntry {  // what an entry brings to a step
  int first, n, pos, slot;
};

// Entry e with its rows; n = 0 for an entry without rows or state (slot -1) and, reported, for one that fits nothing.
__device__ __forceinline__ RecEntry rec_entry(const b200dec_entries& ent, const b200dec_recurrence& rec, int e, int32_t* status) {
  RecEntry x;
  x.first = ent.cu_seqlens ? ent.cu_seqlens[e] : e;
  x.n = ent.cu_seqlens ? ent.cu_seqlens[e + 1] - x.first : 1;
  x.pos = ent.cached_lens[e];
  x.slot = ent.slots[e];
  if (x.n <= 0 || x.slot == -1) {
    x.n = 0;
    return x;
  }
  if (x.slot < 0 || x.slot >= rec.num_slots || x.pos < 0 || x.first < 0 || x.first + x.n > ent.num_rows) {
    if (threadIdx.x == 0 && status) atomicOr(status, B200KV_S_BAD_POSITION);
    x.n = 0;
  }
  return x;
}

struct RecNorm {  // the output norm of the decode kernel
  const float* weight;  // [vdim]; NULL: raw fp32 output
  const void* gate;
  long long gate_stride, out_stride;
  float eps;
};

__host__ __device__ constexpr int rec_round4(int n) { return (n + 3) / 4 * 4; }

__device__ __forceinline__ float ldcg_elem(const uint16_t* p) { return bf16_bits_to_float(__ldcg(p)); }
__device__ __forceinline__ float ldcg_elem(const float* p) { return __ldcg(p); }

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

inline int check_recurrence(const b200dec_recurrence* r, const b200dec_recurrence_in* in, const b200dec_entries* e) {
  if (!r || !in || !e || !r->state || !r->ring || !r->conv_w || !r->neg_a || !r->dt_bias || !in->x || !in->step) return B200KV_E_NULL;
  if (!e->cached_lens || !e->num_decoding || !e->slots || (r->correct && !in->beta)) return B200KV_E_NULL;
  if (e->cu_seqlens && (!e->seq_ids || !e->positions)) return B200KV_E_NULL;
  if (r->num_slots < 1 || r->heads < 1 || r->qk_heads < 1 || r->heads % r->qk_heads || r->dim < 1 || r->vdim < 1 || r->taps < 1)
    return B200KV_E_SHAPE;
  if (r->elem != 2 && r->elem != 4) return B200KV_E_SHAPE;
  if (e->num_entries < 0 || e->num_rows < 0 || e->num_entries > 65535) return B200KV_E_SHAPE;
  const long long qk = (long long)r->qk_heads * r->dim, v = (long long)r->heads * r->vdim;
  if (r->off_q < 0 || r->off_k < 0 || r->off_v < 0 || r->off_q + qk > r->channels || r->off_k + qk > r->channels || r->off_v + v > r->channels)
    return B200KV_E_SHAPE;
  if (!aligned(r->state, 16)) return B200KV_E_ALIGN;
  return B200KV_OK;
}

}  // namespace b200kv
