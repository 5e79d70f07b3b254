/*
 * b200_hybrid_ops.h -- C-ABI of the mixers of hybrid decoders: latent attention over a paged latent cache, gated
 * linear recurrences (Mamba-2, mLSTM) over per-request state slots, and the norms / gates either side of them.
 * Same conventions as b200_paged_ops.h: device pointers, element strides, `stream` is a cudaStream_t, 0 on success.
 *
 * A batch is a list of segments (one per request) of consecutive rows: rows [cu_seqlens[s], cu_seqlens[s+1]) are the
 * new tokens of segment s, seq_lens[s] its length INCLUDING them, so its first row is at position
 * seq_lens[s] - (cu_seqlens[s+1] - cu_seqlens[s]).  A segment that starts at position 0 finds a zero state whatever
 * its slot holds.
 */
#ifndef B200_HYBRID_OPS_H_
#define B200_HYBRID_OPS_H_

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* out[r, :] = table[ids[r], :] widened to fp32 (a 32-bit residual stream). */
int b200_embed_rows(const int32_t* ids, const void* table, float* out, int rows, int vocab, int dim,
                    int64_t out_stride, int dtype, void* stream);

/* out[r, :] = x[row_ids ? row_ids[r] : r, :] / sqrt(mean(x^2) + eps) * (weight + weight_offset); x and weight fp32,
 * out in out_dtype.  weight_offset = 1: weights stored around zero. */
int b200_stream_norm(const float* x, const int64_t* row_ids, const float* weight, void* out, int rows, int dim,
                     int64_t x_stride, int64_t out_stride, float eps, float weight_offset, int out_dtype,
                     void* stream);

/* The element-wise end of a layer's two parallel halves, one launch:
 *   out[r, 0:inner)              = post(gate) * weight * group_norm(y * pre(z))
 *     pre(z) = silu(z) if pre_gate, post(g) = sigmoid(g), or silu(g) with post_silu = 1, if post_gate; group_norm divides each of inner / group_size
 *     parts by its own root mean square (group_size = 0: no norm); weight fp32 or NULL.
 *   out[r, act_offset + i]       = act(act_in[r, i]) (* act_mul[r, i] if given), i in [0, act_dim);
 *     act_kind 0: gelu (erf form), 1: silu, 2: tanh, 3: xIELU, act_a z^2 + z / 2 for z > 0, else act_b (exp(z) - 1 - z) + z / 2.
 *     act_in may be the output columns themselves.
 *   out[r, i] = 0 for the remaining columns below out_cols (alignment padding of the next product's operand).
 * Any of the two halves may be absent (act_dim = 0; y = NULL: the columns below inner are somebody else's). */
typedef struct b200_mixer_finish_args {
  const void* y;
  const void* pre_gate;
  const void* post_gate;
  const float* weight;
  const void* act_in;
  void* out;
  int64_t y_stride, pre_stride, post_stride, act_stride, out_stride;
  int32_t rows, inner, group_size, act_dim, act_offset, out_cols;
  int32_t y_head_dim, y_head_stride; /* y column c is at (c / y_head_dim) * y_head_stride + c % y_head_dim (0: c) */
  float eps;
  int32_t dtype;
  const void* act_mul;
  int64_t mul_stride;
  int32_t act_kind;
  int32_t post_silu;
  float act_a, act_b;
} b200_mixer_finish_args;
int b200_mixer_finish(const b200_mixer_finish_args* a, void* stream);

/* Causal depthwise convolution over segments, then silu if `activation` = 1:
 *   out[t, c] = act(bias[c] + sum_k weight[k, c] * in[t - (taps - 1) + k, c])
 * inputs before the segment come from state[slot, taps-1, channels] (oldest first), which is replaced by the last
 * taps - 1 inputs.  weight fp32 [taps, channels], bias fp32 [channels]. */
int b200_causal_conv(const void* in, const float* weight, const float* bias, void* state, const int32_t* cu_seqlens,
                     const int32_t* seq_lens, const int32_t* slots, void* out, int num_seqs, int max_q_len,
                     int channels, int taps, int64_t in_stride, int64_t out_stride, int activation, int dtype,
                     void* stream);

/* Gated linear recurrence per (segment, head), state S [key_dim, value_dim] in fp32:
 *   kind 0 (Mamba-2): dt = softplus(gate_a + bias_a[h]);
 *       S <- exp(-rate[h] dt) S + dt k v^T;  out = S^T q + skip[h] v;  q / k shared by num_heads / num_groups heads.
 *   kind 1 (mLSTM): i = cap tanh((gate_a + bias_a[h]) / cap), f = logsigmoid(cap tanh((gate_b + bias_b[h]) / cap)),
 *       m' = max(f + m, i); S <- exp(f + m - m') S + exp(i - m') k v^T; n likewise with k alone;
 *       out = S^T q' / (max(|n . q'|, exp(-m')) + 1e-6), q' = q_scale q.
 *   kind 2 (lightning attention): S <- decay[h] S + k v^T;  out = S^T q';  no gates (gate_a, bias_a NULL);
 *       rate[h] = -log(decay[h]), finite, is what the chunked forms use.
 *   kind 3 (RWKV-style): out = (S + diag(u) k v^T)^T q;  then S <- diag(w) S + k v^T  with
 *       w = exp(-exp(gate_a + bias_a)) per head and key channel; gate_a fp32 [rows, heads * key_dim] whatever dtype, bias_a
 *       and u = skip [heads * key_dim]; no groups, q_scale is not applied.
 * silu = 1: q, k and v are taken through silu as they are read (token-by-token form only; for the chunked forms the
 * caller does it beforehand).
 * state [slots, heads, key_dim, value_dim]; mLSTM also norm_state [slots, heads, vtiles, key_dim] and max_state
 * [slots, heads, vtiles] with vtiles = ceil(value_dim / 64): one copy per 64-wide value tile, so that the tiles of a
 * head never wait for one another.
 * Segments of at most seq_limit rows run token by token; longer ones (bf16 only) in chunks of `chunk` rows (what
 * b200_recurrence_chunk says) listed by chunk_seq / chunk_row (segment and first row of every chunk of every longer
 * segment, in order; seq_chunk0[s] = index of segment s's first chunk).  workspace: see
 * b200_recurrence_workspace_bytes. */
#define B200_RECURRENCE_CHUNK 64     /* warp-level tensor cores */
#define B200_RECURRENCE_CHUNK_TC 128 /* tcgen05: key_dim a multiple of 64, at most 512 */
typedef struct b200_recurrence_args {
  const void* q;
  const void* k;
  const void* v;
  const void* gate_a;
  const void* gate_b;
  const float* bias_a;
  const float* bias_b;
  const float* rate;
  const float* skip;
  float* state;
  float* norm_state;
  float* max_state;
  const int32_t* cu_seqlens;
  const int32_t* seq_lens;
  const int32_t* slots;
  const int32_t* chunk_seq;
  const int32_t* chunk_row;
  const int32_t* seq_chunk0;
  void* out;
  void* workspace;
  size_t workspace_bytes;
  int64_t q_stride, k_stride, v_stride, gate_stride, out_stride;
  int32_t kind, dtype, num_tokens, num_seqs, num_heads, num_groups, key_dim, value_dim;
  int32_t num_chunks, chunk, seq_limit;
  float q_scale, gate_cap;
  const float* decay;
  int32_t silu;
} b200_recurrence_args;
size_t b200_recurrence_workspace_bytes(const b200_recurrence_args* a);
/* Rows per chunk of the form that covers this call's type and sizes; 0: token by token only. */
int b200_recurrence_chunk(const b200_recurrence_args* a);
/* Synchronises.  1 if a bounded wait inside a tcgen05 kernel ever ran out (that launch wrote no results), else 0. */
int b200_recurrence_failed(void);
int b200_recurrence(const b200_recurrence_args* a, void* stream);
int b200_recurrence_num_launches(const b200_recurrence_args* a);

/* Hyper-connected residual: a row's stream is num_streams copies of dim columns, fp32 [rows, num_streams, dim].
 *
 * out[r, s, :] = table[ids[r]] (+ sinusoid(positions[r])) for every copy s.  The sinusoid: entry 2i is sin, 2i + 1 cos of
 * positions[r] * f_i, with f_i = freq[2i] + freq[2i + 1] as a high and a low part (positions NULL: none). */
int b200_embed_streams(const int32_t* ids, const void* table, const int32_t* positions, const float* freq, float* out,
                       int rows, int vocab, int dim, int num_streams, int dtype, void* stream);

/* What lies between two sublayers, one launch.  With the result of the sublayer before (y not NULL):
 *   r = y2 ? (rms_norm(y) * y_norm + rms_norm(y2) * y2_norm) / 2 : y;   r *= sigmoid(gate + gate_bias) if gate;
 *   x_t <- sum_s mix[s, t] x_s + out_weight[t] r;                       written back if store
 * and what the sublayer after reads (h not NULL):
 *   u = sum_s in_weight[s] x_s;   h = (u - mean) / sqrt(variance + eps) * norm_weight;
 *   shifted (if given) = h + (h' - h) * shift with h' = previous[slots[r]], zeros for a request's first token
 *   (seq_lens[r] = 1), and previous[slots[r]] <- h; for batches of one row a request only (row r = request r).
 * row_ids: the stream rows to work on (h is packed, y / gate are indexed like the stream); NULL: all.
 * Weights and streams fp32, the rest of dtype. */
typedef struct b200_stream_step_args {
  float* streams;
  const void* y;
  const void* y2;
  const float* y_norm;
  const float* y2_norm;
  const void* gate;
  const float* gate_bias;
  const float* mix;
  const float* out_weight;
  const float* in_weight;
  const float* norm_weight;
  void* h;
  const float* shift;
  void* previous;
  void* shifted;
  const int32_t* slots;
  const int32_t* seq_lens;
  const int64_t* row_ids;
  int64_t y_stride, y2_stride, gate_stride, h_stride, shifted_stride;
  int32_t rows, num_streams, dim, store;
  float eps;
  int32_t dtype;
} b200_stream_step_args;
#define B200_MAX_STREAMS 16
int b200_stream_step(const b200_stream_step_args* a, void* stream);

/* What lies between two sublayers, one launch, fp32 stream x [rows, dim]:
 *   r = y, or with parts > 0 sum_j part_weight[row, j] y[row * parts + j] (+ sigmoid(extra_gate[row]) extra[row]) (+ bias);
 *   x += r / rms(r) * out_norm, without out_norm x += r        (y NULL: no result)
 *   x += table_scale * table[ids[row]], if table (fresh = 1: x starts as that and is not read);  x += add, if add
 *   h = x / rms(x) * in_norm, each of `groups` parts of a row by its own rms (0: one part; h and h32 NULL: nothing follows);
 *       h32: as it is in fp32, h: of dtype
 *   mixes > 0 (batches of one row a request): instead h[s, row, :] = h + (h' - h) * mix_weight[s, :] with h' = mix_state[slots[row],
 *       dim], zeros for a request's first token, which takes h (all fp32; h [mixes, rows, dim] with mix_stride)
 *   h += conv(h) with taps weights [taps, dim] if conv_weight: the earlier inputs come from state[slots[row], taps - 1, dim]
 *   (oldest first; zeros for a request's first tokens, seq_lens[row] counts this one), which takes h in; for batches of
 *   one row a request.
 * row_ids: the stream rows to work on (h is packed, the result is indexed like the stream), x is not written then.
 * Norm, gate and convolution weights fp32; y, extra, h and state of dtype. */
typedef struct b200_residual_step_args {
  float* x;
  const void* y;
  const float* part_weight;
  const void* extra;
  const float* extra_gate;
  const float* out_norm;
  const float* in_norm;
  void* h;
  const float* conv_weight;
  void* state;
  const int32_t* slots;
  const int32_t* seq_lens;
  const int64_t* row_ids;
  int64_t y_stride, extra_stride, gate_stride, h_stride;
  int32_t rows, dim, parts, taps;
  float eps;
  int32_t dtype;
  const float* bias;
  const void* table;
  const int32_t* ids;
  const float* add;
  float* h32;
  const float* mix_weight;
  float* mix_state;
  int64_t mix_stride;
  float table_scale;
  int32_t vocab, fresh, groups, mixes;
} b200_residual_step_args;
int b200_residual_step(const b200_residual_step_args* a, void* stream);

/* Rows mixed with the row before, for batches with portions: out[s, t, :] = h[t] + (h' - h[t]) * weight[s, :] for s < mixes,
 * h' = the row before of the same segment, for its first row state[slot, dim] (zeros for a sequence's first token); the slot takes
 * the segment's last row.  h, weight [mixes, dim] and state fp32; out [mixes, rows, dim] (mix_stride, out_stride) of dtype. */
#define B200_MAX_MIXES 8
int b200_token_mix(const float* h, const float* weight, float* state, const int32_t* cu_seqlens, const int32_t* seq_lens,
                   const int32_t* slots, void* out, int num_seqs, int max_q_len, int dim, int mixes, int64_t h_stride,
                   int64_t out_stride, int64_t mix_stride, int dtype, void* stream);

#define B200_MAX_EXPERTS 1024
/* Routed experts.  b200_expert_route, per row: s = softmax(logits[row, 0:experts]); the `top` experts with the largest
 * s + correction (fp32, NULL: 0; ties to the lower number), best first, go to chosen [rows, top] and their s * scale to
 * weights [rows, top].  over_chosen = 1: the correction is part of the logits, the largest of them are chosen, and the weights are
 * the softmax over the chosen ones alone, times scale. */
int b200_expert_route(const float* logits, int64_t logits_stride, const float* correction, int32_t* chosen, float* weights,
                      int rows, int experts, int top, float scale, int over_chosen, void* stream);

/* The (row, place) pairs p = row * top + place sorted by expert: pairs [rows * top], first [experts + 1] the start of each
 * expert's stretch, tiles [experts + 1] the running count of the stretches' tiles of tile_rows pairs. */
int b200_expert_plan(const int32_t* chosen, int32_t* pairs, int32_t* first, int32_t* tiles, int rows, int experts, int top,
                     int tile_rows, void* stream);

/* Products of all experts at once.  `gated` = 1, the way in:
 *   out[i, n] = silu(w[e, n] . x[pairs[i] / top]) * (w[e, inter + n] . x[pairs[i] / top])   i in e's stretch, n < n_out
 * (w [experts, 2 n_out, k], out [pairs, n_out] in sorted order); 0, the way out:
 *   out[pairs[i], n] = w[e, n] . x[i]                                            (w [experts, n_out, k], x in sorted order).
 * A shared expert that every row takes runs in the same launch (shared_w not NULL): its rows are x (gated) or shared_x, its
 * results shared_out [rows, shared_n_out].  Element strides; rows of w and shared_w are w_stride and shared_w_stride apart.
 * kernel: 0 auto, 1 any type and size, 2 tcgen05 (bf16, whole 8-element units; an odd n_out also writes the column after it).  tile_rows as given to the plan (32, 64 or
 * 128); max_tiles bounds tiles[experts]. */
typedef struct b200_expert_product_args {
  const void* x;
  const void* w;
  void* out;
  const void* shared_x;
  const void* shared_w;
  void* shared_out;
  const int32_t* pairs;
  const int32_t* first;
  const int32_t* tiles;
  int64_t x_stride, w_stride, out_stride, shared_x_stride, shared_w_stride, shared_out_stride;
  int32_t rows, experts, top, n_out, k, shared_n_out, shared_k, tile_rows, max_tiles, gated, dtype, kernel;
} b200_expert_product_args;
int b200_expert_product(const b200_expert_product_args* a, void* stream);
/* Synchronises.  1 if the tcgen05 kernel ever found a plan that does not fit together or a bounded wait inside it ran out (that
 * launch's results are invalid), else 0. */
int b200_expert_product_failed(void);

/* Before latent attention, per row: the latent is normed (weight fp32, plain), the shared key part is rotated
 * (interleaved pairs), both go to the latent cache row slot_mapping[t]:
 * [latent kv_rank | key part rot_dim]; the rotated part of every query head goes to
 * q_out[t, h, rot_offset + ...], and with copy_nope the unrotated part to q_out[t, h, 0 : dim), columns from
 * rot_offset + rot_dim to q_cols zeroed. */
typedef struct b200_latent_prep_args {
  const void* q;
  const void* down;
  const float* norm_weight;
  const int32_t* positions;
  const int64_t* slot_mapping;
  const float* inv_freq; /* [rot_dims / 2], base^(-2i/rot_dims) */
  void* cache;
  void* q_out;
  int64_t q_stride, down_stride, q_out_stride;
  int64_t num_slots;
  int32_t num_tokens, heads, dim, rot_dim, rot_dims, kv_rank;
  int32_t q_cols, rot_offset, copy_nope;
  float eps;
  int32_t dtype;
} b200_latent_prep_args;
int b200_latent_prep(const b200_latent_prep_args* a, void* stream);

/* Before attention with rotated, then normed heads, per row: the interleaved pairs (2i, 2i + 1) of the first rot_dims
 * dimensions of every query and key head are turned by positions[t] * f_i and scaled by rot_factor, with f_i = freq[2i] +
 * freq[2i + 1] as a high and a low part; the head is divided by its root mean square; a query head also takes
 * q_weight[h] (fp32, NULL: 1).  With q_norm / k_norm (fp32 [dim]) queries / keys are multiplied by them, with norm_values a
 * value head is divided by its root mean square, and with temp_coef a query is multiplied by
 * 1 + temp_coef ln(floor((positions[t] + 1) / temp_every) + 1).  Queries are updated in place, keys and values go to cache row slot_mapping[t] (negative or out of
 * range: padding, nothing is cached). */
typedef struct b200_rope_norm_cache_args {
  void* q;
  const void* k;
  const void* v;
  const float* q_weight;
  const float* freq; /* [rot_dims / 2][2] */
  const int32_t* positions;
  const int64_t* slot_mapping;
  void* key_cache; /* [num_blocks, block_size, kv_heads, dim], rows contiguous */
  void* value_cache;
  int64_t q_stride, k_stride, v_stride;
  int64_t k_block_stride, k_token_stride, v_block_stride, v_token_stride, num_blocks;
  int32_t num_tokens, heads, kv_heads, dim, vdim, rot_dims, block_size;
  float rot_factor, eps;
  int32_t dtype;
  const float* q_norm;
  const float* k_norm;
  float temp_coef, temp_every;
  int32_t norm_values;
} b200_rope_norm_cache_args;
int b200_rope_norm_cache(const b200_rope_norm_cache_args* a, void* stream);

/* y[t, h, n] = sum_k w[h, n, k] x[t, h, k], times sigmoid(gate[t, h * n_dim + n]) if gate: the per-head products of
 * latent attention (queries into the latent space, latent outputs into value space). */
typedef struct b200_head_linear_args {
  const void* x;
  const void* w;
  const void* gate;
  void* y;
  int64_t x_stride, x_head_stride, y_stride, y_head_stride, gate_stride;
  int32_t rows, heads, n, k, dtype;
} b200_head_linear_args;
int b200_head_linear(const b200_head_linear_args* a, void* stream);

/* Latent attention in the latent space: every query head attends over the same cached rows
 * [latent kv_rank | key part rot_dim]; values are the latents.  q [T, heads, kv_rank + rot_dim], out
 * [T, heads, kv_rank].  Only segments of at most max_q_len rows are computed.  window <= 0: none.
 * kernel: 0 auto, 1 any type and size, 2 warp-level tensor cores, 3 tcgen05. */
typedef struct b200_latent_attn_args {
  const void* q;
  const void* cache;
  const int32_t* block_tables;
  const int32_t* seq_lens;
  const int32_t* cu_seqlens;
  void* out;
  void* workspace;
  size_t workspace_bytes;
  int64_t q_stride, out_stride;
  int64_t num_slots;
  int32_t num_tokens, num_seqs, heads, kv_rank, rot_dim, block_size, max_blocks_per_seq, max_seq_len, window;
  int32_t max_q_len;
  int32_t dtype, kernel, force_splits;
  float scale;
} b200_latent_attn_args;
size_t b200_latent_attention_workspace_bytes(const b200_latent_attn_args* a);
int b200_latent_attention_num_launches(const b200_latent_attn_args* a);
int b200_latent_attention(const b200_latent_attn_args* a, void* stream);
/* Synchronises.  1 if a bounded wait inside the kernel ever ran out (that launch wrote no results), else 0. */
int b200_latent_attention_failed(void);

/* Rows [first[i], first[i] + count[i]) of request i's cached latents, gathered from the pages into consecutive rows
 * of out [rows, kv_rank + rot_dim] starting at out_row[i] (the operand of the products that expand keys and values);
 * rows between out_row[i] + count[i] and the next multiple of `pad` are zeroed. */
int b200_latent_gather(const void* cache, const int32_t* block_tables, const int32_t* first, const int32_t* count,
                       const int32_t* out_row, void* out, int num_seqs, int max_count, int width, int block_size,
                       int max_blocks_per_seq, int64_t num_slots, int pad, int dtype, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* B200_HYBRID_OPS_H_ */
