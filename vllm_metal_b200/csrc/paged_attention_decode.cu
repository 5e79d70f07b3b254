// Host side of the tensor-core decode kernel and its forms for keys and values of one size (64 or 128).
#include "paged_attention_decode.cuh"

namespace b200 {

static int log2_exact_i(int v) {
  int s = 0;
  while ((1 << s) < v) ++s;
  return (1 << s) == v ? s : -1;
}

// The forms that were there for keys and values of one size; everything else (and 16-bit-wide weights) is bf16 only.
static bool plain_form(const b200_paged_attn_args& a) {
  return (a.head_dim == 64 || a.head_dim == 128) && value_dim(a) == a.head_dim && !a.wide_weights && keep_first(a) == 0 &&
         !a.slopes;
}

bool decode_mma_supported(const b200_paged_attn_args& a) {
  if (a.dtype != B200_BF16 && a.dtype != B200_F16) return false;
  const ValueStrides vs = value_strides(a);
  const int dk = a.head_dim, dv = value_dim(a);
  if (!plain_form(a)) {
    const bool same = dk == dv && (dk == 64 || dk == 128);  // fp16 and window batches: as without wide weights
    if (a.dtype != B200_BF16 && !same) return false;
    if (dk % 8 || dv % 8 || dk > 256 || dv > 256 || (a.window_seqlen_q > 1 && !same)) return false;
  }
  // kept first positions: bf16, one row a CTA (window batches know one visible stretch a row)
  if (keep_first(a) > 0 && (a.dtype != B200_BF16 || a.window_seqlen_q > 1)) return false;
  if (a.slopes && (a.dtype != B200_BF16 || a.window_seqlen_q > 1)) return false;  // the same for a distance bias
  const int G = a.num_q_heads / a.num_kv_heads;
  if (G < 1 || G > 16) return false;
  if (log2_exact_i(a.block_size) < 0) return false;
  if (a.kv_block_stride % 8 || a.kv_token_stride % 8 || a.kv_head_stride % 8) return false;
  if (vs.block % 8 || vs.token % 8 || vs.head % 8) return false;
  if (a.q_stride % 2) return false;
  if (((uintptr_t)a.key_cache | (uintptr_t)a.value_cache) % 16) return false;
  if ((uintptr_t)a.query % 4) return false;
  // row offsets are carried as 32-bit counts of 16-byte units
  if ((a.num_blocks * a.kv_block_stride) / 8 >= 0xFFFFFFF0ll || (a.num_blocks * vs.block) / 8 >= 0xFFFFFFF0ll) return false;
  return true;
}

static bool wide_form(const b200_paged_attn_args& a) {
  return !plain_form(a) && a.dtype == B200_BF16 && a.window_seqlen_q <= 1;
}

int decode_mma_ctas_per_sm(const b200_paged_attn_args& a) {
  return decode_ctas_per_sm(decode_key_width(a.head_dim), decode_value_width(value_dim(a)));
}

template <typename T, int D, int STAGES>
static int launch_one(const DecodeParams& p, dim3 grid, cudaStream_t st) {
  if (p.win_rows > 1) return launch_decode_form<T, D, D, STAGES, true, false>(p, grid, st);
  return launch_decode_form<T, D, D, STAGES, false, false>(p, grid, st);
}

// Window mode (a `window_seqlen_q` hint > 1): query rows of one sequence that share a CTA -- the MMA rows the GQA
// group leaves free.  1 = per-row dispatch.
int decode_window_rows(const b200_paged_attn_args& a) {
  if (a.window_seqlen_q <= 1) return 1;
  const int G = a.num_q_heads / a.num_kv_heads;
  const int r = G > 0 ? 16 / G : 1;
  return r < 1 ? 1 : (r > a.window_seqlen_q ? a.window_seqlen_q : r);
}

int launch_decode_mma(const b200_paged_attn_args& a, const SplitWorkspace* ws, cudaStream_t st, int skip_qlen) {
  DecodeParams p{};
  p.out = a.out;
  p.query = a.query;
  p.key_cache = (const uint8_t*)a.key_cache;
  p.value_cache = (const uint8_t*)a.value_cache;
  p.block_tables = a.block_tables;
  p.seq_lens = a.seq_lens;
  p.cu_seqlens_q = a.cu_seqlens_q;
  p.sinks = a.sinks;
  p.slopes = a.slopes;
  p.num_seqs = a.num_seqs;
  p.num_q_heads = a.num_q_heads;
  p.num_kv_heads = a.num_kv_heads;
  p.group = a.num_q_heads / a.num_kv_heads;
  p.block_shift = log2_exact_i(a.block_size);
  p.max_blocks_per_seq = a.max_blocks_per_seq;
  p.sliding_window = a.sliding_window;
  p.keep_first = keep_first(a);
  p.q_stride = a.q_stride;
  p.out_stride = a.out_stride;
  p.block_stride16 = (uint32_t)(a.kv_block_stride / 8);
  p.token_stride16 = (uint32_t)(a.kv_token_stride / 8);
  const ValueStrides vs = value_strides(a);
  p.v_block_stride16 = (uint32_t)(vs.block / 8);
  p.v_token_stride16 = (uint32_t)(vs.token / 8);
  p.head_stride_bytes = a.kv_head_stride * 2;
  p.v_head_stride_bytes = vs.head * 2;
  p.head_dim = a.head_dim;
  p.value_dim = value_dim(a);
  p.num_blocks = a.num_blocks;
  p.scale = a.scale;
  p.softcap = a.softcap;
  p.partitioned = ws != nullptr;
  p.ws = SplitWorkspace{};
  if (ws) p.ws = *ws;
  p.ws.skip_qlen = skip_qlen;
  p.ws.out_f16 = out_is_f16(a);
  p.ws.denom_eps = denom_eps(a);
  dim3 grid(a.num_kv_heads, a.num_q_tokens, ws ? ws->num_partitions : 1);
  p.win_rows = skip_qlen > 0 ? 1 : decode_window_rows(a);
  p.win_subs = 1;
  if (p.win_rows > 1) {  // one CTA per (sequence, sub-window of win_rows rows); paged_ops.cpp:508-515
    p.win_subs = (a.window_seqlen_q + p.win_rows - 1) / p.win_rows;
    grid.y = (unsigned)(a.num_seqs * p.win_subs);
  }
  if (p.keep_first > 0) return p.group <= 8 ? launch_decode_kept_packed(p, grid, st) : launch_decode_kept(p, grid, st);
  if (wide_form(a)) return p.group <= 8 ? launch_decode_wide_packed(p, grid, st) : launch_decode_wide(p, grid, st);
  if (a.dtype == B200_BF16) {
    if (a.head_dim == 128) return launch_one<__nv_bfloat16, 128, 3>(p, grid, st);
    return launch_one<__nv_bfloat16, 64, 4>(p, grid, st);
  }
  if (a.head_dim == 128) return launch_one<__half, 128, 3>(p, grid, st);
  return launch_one<__half, 64, 4>(p, grid, st);
}

}  // namespace b200
