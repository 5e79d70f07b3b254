// Internal interface between the paged-attention router and its kernels.
#pragma once
#include "common.cuh"

namespace b200 {

// Split-KV scratch layout (fp32 partials; SURVEY.md appendix A.4 -- the
// reference keeps tmp_out in the query dtype, paged_ops.cpp:647-653):
//   tmp_out  float [T, H_q, P, D]   un-normalised partial numerators
//   max_l2   float [T, H_q, P]      running max in the log2 domain
//   exp_sum  float [T, H_q, P]      sum of 2^(s - max)
struct SplitWorkspace {
  float* tmp_out;
  float* max_l2;
  float* exp_sum;
  int num_partitions;  // P
  int partition_size;  // tokens
  int skip_qlen;       // > 0: rows of sequences with q_len >= skip_qlen belong to the tile kernel (left untouched here)
  int out_f16;         // bf16 call whose `out` buffer is fp16: store the bf16-rounded value as fp16 (args.out_dtype)
  float denom_eps;     // added to the softmax denominator (args.plain_softmax)
};

// Values may have a head size and strides of their own.
inline int value_dim(const b200_paged_attn_args& a) { return a.value_dim > 0 ? a.value_dim : a.head_dim; }
struct ValueStrides {
  int64_t block, token, head;
};
inline ValueStrides value_strides(const b200_paged_attn_args& a) {
  if (a.v_token_stride > 0) return {a.v_block_stride, a.v_token_stride, a.v_head_stride};
  return {a.kv_block_stride, a.kv_token_stride, a.kv_head_stride};
}
// Kept first positions matter beside a window only; no row has more than max_seq_len.
inline int keep_first(const b200_paged_attn_args& a) {
  return a.sliding_window < 0 ? 0 : a.keep_first < a.max_seq_len ? a.keep_first : a.max_seq_len;
}
inline float denom_eps(const b200_paged_attn_args& a) { return a.plain_softmax ? 0.f : 1e-6f; }

// One output element: rounded to the call's dtype T; with out_f16 (T = bf16) that value is stored as fp16 -- exact
// below 65504 -- so the o_proj that follows (fp16 tensor-core operands) needs no cast launch.
template <typename T>
__device__ __forceinline__ void store_out(T* row, int d, float v, int out_f16) {
  const T t = from_float<T>(v);
  if (out_f16) reinterpret_cast<__half*>(row)[d] = __float2half_rn(fminf(fmaxf(to_float(t), -65504.f), 65504.f));
  else row[d] = t;
}

inline size_t split_workspace_bytes(int64_t T, int64_t Hq, int64_t P, int64_t D) {
  return (size_t)(T * Hq * P * (D + 2)) * sizeof(float);
}

inline SplitWorkspace carve_workspace(void* ws, int64_t T, int64_t Hq, int64_t P, int64_t D,
                                      int partition_size) {
  SplitWorkspace w;
  w.tmp_out = reinterpret_cast<float*>(ws);
  w.max_l2 = w.tmp_out + T * Hq * P * D;
  w.exp_sum = w.max_l2 + T * Hq * P;
  w.num_partitions = (int)P;
  w.partition_size = partition_size;
  w.skip_qlen = 0;
  w.out_f16 = 0;
  w.denom_eps = 1e-6f;
  return w;
}

// Row (token) -> sequence lookup; reference find_seq_idx,
// pagedattention.metal:772-784 (binary search over cu_seqlens_q).
__device__ __forceinline__ int find_seq_idx(const int32_t* __restrict__ cu, int num_seqs, int t) {
  int lo = 0, hi = num_seqs;  // invariant: cu[lo] <= t < cu[hi]
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid;
  }
  return lo;
}

// Per-row KV range.  `eff` = number of KV positions row t may see
// (pagedattention.metal:913); with a sliding window W only [eff-W, eff) is kept
// (:1129-1133).  Split-KV partitions are laid out from `base` (the window start
// rounded down to a 16-token tile), so windowed rows need ceil((W+15)/psize)
// partitions instead of ceil(max_seq_len/psize): pages wholly outside the window
// are never touched (the reference iterates and masks them).
//
// Kept first positions [0, keep_first) come ahead of the window: the 16-token tiles that hold them and lie wholly before
// `base` are `kept` tiles.  A row's tiles are then numbered 0 .. without the gap between the two stretches; `gap` is
// what a token counted that way has to be moved by once it is past the kept tiles (token_at), and partitions are laid
// out over these numbers.
struct RowInfo {
  int seq, eff, beg, base;
  int kept, gap;
  __device__ __forceinline__ int span() const { return eff - base + kept * 16; }
  __device__ __forceinline__ int token_at(int v) const { return v < kept * 16 ? v : v + gap; }
};
__device__ __forceinline__ RowInfo row_info(const int32_t* __restrict__ cu,
                                            const int32_t* __restrict__ seq_lens, int num_seqs,
                                            int t, int sliding_window, int keep_first, int skip_qlen = 0) {
  RowInfo r;
  r.seq = find_seq_idx(cu, num_seqs, t);
  const int q_start = cu[r.seq];
  const int q_len = cu[r.seq + 1] - q_start;
  r.eff = seq_lens[r.seq] - q_len + (t - q_start) + 1;
  if (skip_qlen > 0 && q_len >= skip_qlen) r.eff = 0;  // mixed batch: the tile kernel owns this sequence
  r.beg = 0;
  r.base = 0;
  r.kept = 0;
  if (sliding_window >= 0) {
    r.beg = max(0, r.eff - sliding_window);
    r.base = r.beg & ~15;
    r.kept = min((keep_first + 15) >> 4, r.base >> 4);
  }
  r.gap = r.base - r.kept * 16;
  return r;
}

// Launchers implemented in paged_attention_generic.cu / paged_attention_decode.cu.
// `ws == nullptr` => single pass.
int launch_generic(const b200_paged_attn_args& a, const SplitWorkspace* ws, cudaStream_t st, int skip_qlen = 0);
inline int out_is_f16(const b200_paged_attn_args& a) { return a.out_dtype == B200_F16 && a.dtype == B200_BF16 ? 1 : 0; }
bool decode_mma_supported(const b200_paged_attn_args& a);
int decode_mma_ctas_per_sm(const b200_paged_attn_args& a);
int launch_decode_mma(const b200_paged_attn_args& a, const SplitWorkspace* ws, cudaStream_t st, int skip_qlen = 0);
int decode_window_rows(const b200_paged_attn_args& a);  // > 1: window mode (query rows of one sequence per CTA)
int launch_split_reduce(const b200_paged_attn_args& a, const SplitWorkspace& ws, cudaStream_t st);
// Tile kernel (paged_attention_prefill.cu): sequences with q_len >= min_qlen, one CTA per (128-row Q tile, q head).
bool prefill_tc_supported(const b200_paged_attn_args& a);
int launch_prefill_tc(const b200_paged_attn_args& a, int min_qlen, cudaStream_t st);

}  // namespace b200
