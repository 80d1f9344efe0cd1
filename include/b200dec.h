/*
 * b200dec.h — C ABI of the decoder ops that work in the model's own precision: a paged KV cache of unquantised
 * rows (bf16 or fp32, key and value sizes free of one another), partial rotary positions, attention over that cache,
 * a 32-bit residual stream, and a mixture of experts.
 *
 * Built beside b200kv.h (the int8-cache attention path) and with its conventions: device pointers, strides in
 * elements, no allocation and no synchronisation, grids from shape arguments only (every call can be captured in a CUDA
 * graph), B200KV_* return codes (negative: nothing was launched) and status bits (device-side inconsistencies: the
 * access is skipped).  `elem` is the element size of the model's precision: 2 = bf16, 4 = fp32.
 */
#ifndef B200DEC_H
#define B200DEC_H

#include "b200kv.h"

#ifdef __cplusplus
extern "C" {
#endif

/* One layer's cache.  k [num_pages, kv_heads, page_size, k_row], v [num_pages, kv_heads, page_size, v_row], contiguous;
 * k_row / v_row are k_dim / v_dim rounded up to a multiple of 8, and the channels behind k_dim / v_dim are zero. */
typedef struct b200dec_cache {
  void* k;
  void* v;
  int32_t num_pages, kv_heads, page_size;
  int32_t k_dim, v_dim, k_row, v_row;
  int32_t elem;
} b200dec_cache;

/* Which (entry, position) each packed row of a step is.
 * seq_ids and positions set: a step with prompt portions; row r belongs to entry seq_ids[r] and sits at positions[r].
 * Both NULL: a pure decode step; row r is the new token of entry r at position cached_lens[r], rows from *num_decoding
 * on are idle. */
typedef struct b200dec_rows {
  const int32_t* seq_ids;
  const int32_t* positions;
  const int32_t* cached_lens;
  const int32_t* num_decoding;
  int32_t num_rows;
} b200dec_rows;

/* x[r] = fp32(table[ids[r]]), xb[r] = table[ids[r]] (xb may be NULL).  Ids outside [0, vocab) read row 0 and set
 * B200KV_S_BAD_POSITION. */
int b200dec_embed(const void* table, int32_t elem, const int32_t* ids, float* x, void* xb, int32_t num_rows, int32_t width,
                  int32_t vocab, int32_t* status, void* stream);

/* Residual update in the norm-after-the-sum arrangement, 32-bit:
 *   s = alpha * x[r] + sum_j delta[index[r * top + j]]       (index NULL: delta[r]; delta NULL: s = alpha * x[r])
 *   y = s / sqrt(mean(s^2) + eps) * weight
 * x_out[r] = y (fp32; may be x itself, may be NULL), xb_out[r] = y in the model's precision (may be NULL).
 * delta and xb_out have element size `elem`; weight is fp32 [width].  `zero` (may be NULL): int32 [num_zero], cleared
 * by the first block, for the kernel that counts into it next. */
int b200dec_scaled_add_norm(const float* x, const void* delta, const int32_t* index, int32_t top, int32_t elem, const float* weight,
                            float alpha, float eps, float* x_out, void* xb_out, int32_t num_rows, int32_t width, int32_t* zero,
                            int32_t num_zero, void* stream);

/* Rotary positions and unit norm of packed projection rows, and the write of keys and values into the cache.
 * qkv row r: q [heads, k_dim] | k [kv_heads, k_dim] | v [kv_heads, v_dim], consecutive, row stride qkv_stride.  With
 * write_kv = 0 the row holds q only and the cache is untouched (a layer that attends another layer's cache).
 * cos_sin fp32 [positions, half, 2] (cos, sin per pair, multiplier included): channel i < half is paired with i + half;
 * half may be 0.  After the rotation, with unit_norm != 0, q and k heads are divided by sqrt(mean(.^2) + eps).
 * q_out [num_rows, heads, k_row], padding channels zeroed. */
int b200dec_rope_write(const void* qkv, int64_t qkv_stride, const b200dec_rows* rows, const b200dec_cache* cache,
                       const b200kv_table* table, const float* cos_sin, int32_t table_len, int32_t half, int32_t heads,
                       int32_t write_kv, int32_t unit_norm, float eps, void* q_out, int32_t* status, void* stream);

/* Causal attention of packed rows over the cache (the rows' own keys already written): row at position p attends
 * positions 0..p.  out [num_rows, heads, v_dim].  Any sizes up to k_dim, v_dim <= 1024; CUDA cores, 32-bit throughout. */
int b200dec_attn_rows(const void* q, const b200dec_cache* cache, const b200kv_table* table, const b200dec_rows* rows, int32_t heads,
                      float scale, void* out, int32_t* status, void* stream);

/* The product path for bf16 caches with k_dim, v_dim <= 128 (else B200KV_E_SHAPE): entries b < *num_decoding, query row b,
 * at position cached_lens[b].  Split over a persistent grid, pieces merged by the last arriver; `workspace` zero-filled
 * once and left so.  zero_idle != 0: rows b in [*num_decoding, B) of `out` are zeroed (a step without prompt portions). */
size_t b200dec_decode_attn_workspace(int32_t B, int32_t heads, int32_t kv_heads, int32_t v_dim, int32_t sm_count);
int b200dec_decode_attn(const void* q, const b200dec_cache* cache, const b200kv_table* table, const int32_t* cached_lens,
                        const int32_t* num_decoding, int32_t B, int32_t heads, float scale, void* out, int32_t zero_idle,
                        void* workspace, size_t workspace_bytes, int32_t sm_count, int32_t* status, void* stream);

/* Prompt portions on tcgen05, bf16 cache with k_dim, v_dim <= 128 and page_size a multiple of 16: query tiles of 128 rows
 * as in b200kv_prefill_attn (tile_start, seq_ids, cu_seqlens), keys and values read from the cache by page. */
int b200dec_prefill_attn(const void* q, const b200dec_cache* cache, const b200kv_table* table, const int32_t* seq_ids,
                         const int32_t* cu_seqlens, const int32_t* cached_lens, const int32_t* tile_start, int32_t num_tiles,
                         int32_t block_m, int32_t num_rows, int32_t heads, float scale, void* out, int32_t* status, void* stream);

/* ---- mixture of experts.  Tokens are routed (router), laid out by expert (dispatch), and pass two grouped products; the
 * sum over a token's experts is b200dec_scaled_add_norm with index = slots, top.
 *
 * router: scores = sigmoid(router_w x), 32-bit, router_w bf16 [experts, width], x fp32 [num_rows, width]; the `top` largest
 * scores of a row (ties: smaller expert id).  ids, ranks int32 [num_rows * top], scores fp32 [num_rows * top];
 * counts int32 [experts] must be zero on entry; ranks number an expert's tokens in arrival order. */
int b200dec_router(const float* x, const void* router_w, int32_t num_rows, int32_t width, int32_t experts, int32_t top, int32_t* ids,
                   float* scores, int32_t* ranks, int32_t* counts, void* stream);
/* dispatch: copies row r of xb to the places of its experts in x_sorted [num_rows * top, width] (experts' tokens
 * consecutive), slots[r * top + j] = that place, score_sorted[place] = its score, and cuts every expert's run into tiles of
 * at most tile_rows rows: tiles int32 [1 + 3 * max_tiles] = count, then (expert, first row, rows) each, with
 * max_tiles = num_rows * top / tile_rows + min(experts, num_rows * top). */
int b200dec_dispatch(const void* xb, int32_t elem, const int32_t* ids, const float* scores, const int32_t* ranks, const int32_t* counts,
                     int32_t num_rows, int32_t width, int32_t experts, int32_t top, int32_t tile_rows, void* x_sorted,
                     float* score_sorted, int32_t* slots, int32_t* tiles, int32_t max_tiles, void* stream);
/* grouped product: y[row] = W_e x[row] for the rows of every tile; w [experts, out_rows, width].
 * act = 0: y [rows, out_rows].  act = 1: W_e's rows alternate gate, up; with the row's score s,
 *   g = min(s * gate . x, limit), u = clamp(s * up . x, -limit, limit), y = g * sigmoid(slope * g) * (u + 1),
 * y [rows, out_rows / 2].  variant 0: tcgen05 for bf16 when width and the row strides allow TMA (width % 8 == 0),
 * variant 1: CUDA cores, any sizes, fp32 or bf16. */
int b200dec_grouped_linear(const void* x, const void* w, int32_t elem, const int32_t* tiles, int32_t max_tiles, int32_t tile_rows,
                           int32_t total_rows, int32_t experts, int32_t out_rows, int32_t width, const float* score_sorted,
                           int32_t act, float limit, float slope, void* y, int32_t sm_count, int32_t variant, int32_t* status, void* stream);

/* ---- attention with a sliding window, a sink and an output gate: the three kernels above with options.
 * window > 0: the row at position i sees positions j with 0 <= i - j < window (0: all j <= i).
 * sink fp32 [heads] (may be NULL): exp(sink[h]) joins the softmax denominator of head h, unscaled.
 * gate (may be NULL), element size as the cache's: head h of row r is multiplied by sigmoid(gate[r * gate_stride + h]).
 * out_scale multiplies the result; out rows are out_stride elements apart (0: heads * v_dim; a multiple of 8 otherwise). */
typedef struct b200dec_attn_options {
  int32_t window;
  const float* sink;
  const void* gate;
  int64_t gate_stride;
  float out_scale;
  int64_t out_stride;
} b200dec_attn_options;

int b200dec_attn_rows_opt(const void* q, const b200dec_cache* cache, const b200kv_table* table, const b200dec_rows* rows, int32_t heads,
                          float scale, const b200dec_attn_options* opt, void* out, int32_t* status, void* stream);
int b200dec_decode_attn_opt(const void* q, const b200dec_cache* cache, const b200kv_table* table, const int32_t* cached_lens,
                            const int32_t* num_decoding, int32_t B, int32_t heads, float scale, const b200dec_attn_options* opt, void* out,
                            int32_t zero_idle, void* workspace, size_t workspace_bytes, int32_t sm_count, int32_t* status, void* stream);
int b200dec_prefill_attn_opt(const void* q, const b200dec_cache* cache, const b200kv_table* table, const int32_t* seq_ids,
                             const int32_t* cu_seqlens, const int32_t* cached_lens, const int32_t* tile_start, int32_t num_tiles,
                             int32_t block_m, int32_t num_rows, int32_t heads, float scale, const b200dec_attn_options* opt, void* out,
                             int32_t* status, void* stream);

/* RMS norm of the whole query projection and of the whole key projection (q_norm fp32 [heads * k_dim], k_norm fp32
 * [kv_heads * k_dim]), then rotary positions on channel pairs (2i, 2i + 1), i < half, then the write as in b200dec_rope_write
 * (write_kv = 1).  cos_sin as there. */
int b200dec_norm_rope_write(const void* qkv, int64_t qkv_stride, const b200dec_rows* rows, const b200dec_cache* cache,
                            const b200kv_table* table, const float* q_norm, const float* k_norm, float eps, const float* cos_sin,
                            int32_t table_len, int32_t half, int32_t heads, void* q_out, int32_t* status, void* stream);

/* Residual update with the norm on the sublayer's output: x[r] += mult * (y[r] / sqrt(mean(y[r]^2) + eps) * weight), 32-bit;
 * xb (may be NULL) receives the new row in the model's precision.  y has element size `elem`. */
int b200dec_norm_add(float* x, const void* y, int32_t elem, const float* weight, float mult, float eps, void* xb, int32_t num_rows,
                     int32_t width, void* stream);

/* out[r, c] = silu(gate_up[r, c]) * gate_up[r, ff + c] */
int b200dec_silu_mul(const void* gate_up, int64_t stride, int32_t elem, void* out, int64_t out_stride, int32_t num_rows, int32_t ff,
                     void* stream);

/* ---- recurrent layers: a matrix state per request slot and head, 32-bit.
 * One token of one head (query/key head of head h: h / (heads / qk_heads)):
 *   S <- decay * S;  u = beta (v - S^T k)  [correct]  or  step * v;  S <- S + k u^T;  o = S^T q (+ skip v)
 * q, k, v pass a causal convolution of `taps` taps per channel and silu first; with unit_norm q and k are then divided by
 * sqrt(sum(.^2) + unit_eps); q is multiplied by q_scale.  step = softplus(step_in + dt_bias), decay = exp(neg_a[h] step):
 * one per head, or with channel_decay one per head and key channel (the rows of S); beta = sigmoid(beta_in).
 * state fp32 [num_slots, heads, dim, round4(vdim)]; ring [num_slots, taps, channels] (element size elem): the convolution's
 * raw inputs, position p at p % taps.  A request at position 0 starts from zero whatever its slot holds. */
typedef struct b200dec_recurrence {
  float* state;
  void* ring;
  const float* conv_w; /* [taps, channels], last row: the current token */
  const float* conv_b; /* [channels] or NULL */
  const float* neg_a;  /* [heads] */
  const float* dt_bias; /* [heads], or [heads * dim] with channel_decay */
  const float* skip;   /* [heads] or NULL */
  int32_t num_slots, heads, qk_heads, dim, vdim, taps, elem;
  int32_t channels, off_q, off_k, off_v; /* first convolution channel of q, k [qk_heads * dim] and v [heads * vdim] */
  int32_t channel_decay, correct, unit_norm;
  float unit_eps, q_scale;
} b200dec_recurrence;

/* A step's projection rows: x [channels] (the convolution's inputs), step [heads or heads * dim], beta [heads] (NULL without
 * `correct`), row strides in elements. */
typedef struct b200dec_recurrence_in {
  const void* x;
  const void* step;
  const void* beta;
  int64_t x_stride, step_stride, beta_stride;
} b200dec_recurrence_in;

/* A step's entries: rows cu_seqlens[e] .. cu_seqlens[e + 1] of entry e, which continues slot slots[e] at position
 * cached_lens[e]; the first *num_decoding entries bring one token each.  cu_seqlens, seq_ids, positions NULL: pure decode,
 * row e = entry e.  An entry with slot -1 (padding of a step) is passed over; its output rows are left as they are. */
typedef struct b200dec_entries {
  const int32_t* cu_seqlens;
  const int32_t* cached_lens;
  const int32_t* num_decoding;
  const int32_t* slots;
  const int32_t* seq_ids;
  const int32_t* positions;
  int32_t num_entries, num_rows;
} b200dec_entries;

/* The first *num_decoding rows, convolution and state in one kernel.  norm_w NULL: out fp32 [rows, heads * vdim] = o.
 * Otherwise out (element size elem, row stride out_stride) = o / sqrt(mean over vdim(o^2) + eps) * norm_w[vdim] *
 * sigmoid(gate) with gate rows [heads * vdim].  Rows from *num_decoding on of a pure decode step are zeroed.
 * variant 0: states pass through shared memory on a persistent grid where they fit it (else as 1); 1: any size. */
int b200dec_recurrence_decode(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const b200dec_entries* ent,
                              const float* norm_w, float eps, const void* gate, int64_t gate_stride, void* out, int64_t out_stride,
                              int32_t variant, int32_t sm_count, int32_t* status, void* stream);
/* Rows from *num_decoding on: silu(convolution) of every channel, conv_out [rows, channels rounded up to 8]. */
int b200dec_conv_rows(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const b200dec_entries* ent, void* conv_out,
                      int32_t* status, void* stream);
/* Entries from *num_decoding on, token after token from conv_out: out fp32 [rows, heads * vdim]; the slots' states and rings
 * are left at the portions' ends.  dim <= 1024. */
int b200dec_recurrence_scan(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const void* conv_out,
                            const b200dec_entries* ent, float* out, int32_t* status, void* stream);
/* The same for the delta rule with channel decay and without skip (dim <= 256), eight tokens at a time, 32-bit throughout;
 * workspace 128-byte aligned, its size 0 where this form does not apply. */
size_t b200dec_recurrence_blocked_workspace(const b200dec_recurrence* rec, const b200dec_entries* ent);
int b200dec_recurrence_blocked(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const void* conv_out,
                               const b200dec_entries* ent, float* out, void* workspace, size_t workspace_bytes, int32_t* status,
                               void* stream);
/* The same for a state-space layer of a bf16 model (one decay per head, dim <= 128, sizes and offsets multiples of 8), sixteen
 * tokens at a time on the tensor cores; workspace 16-byte aligned, its size 0 where this form does not apply. */
size_t b200dec_state_space_chunked_workspace(const b200dec_recurrence* rec);
int b200dec_state_space_chunked(const b200dec_recurrence* rec, const b200dec_recurrence_in* in, const void* conv_out,
                                const b200dec_entries* ent, float* out, void* workspace, size_t workspace_bytes, int32_t sm_count,
                                int32_t* status, void* stream);
/* out[r] (element size elem) = out_scale * norm(o[r] (* silu(gate)  if gate_first)) * weight (* sigmoid(gate) otherwise), the norm
 * taken over `parts` equal parts of the row of `len` each by itself; weight fp32 [weight_len], repeated.  */
int b200dec_gated_norm(const float* o, const void* gate, int64_t gate_stride, int32_t gate_first, int32_t elem, const float* weight,
                       int32_t weight_len, float eps, float out_scale, void* out, int64_t out_stride, int32_t num_rows, int32_t len,
                       int32_t parts, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* B200DEC_H */
