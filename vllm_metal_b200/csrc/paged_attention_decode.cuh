// Bandwidth path of paged attention: GQA-shared, split-KV, tensor-core decode.
//
// One CTA per (kv head, query row, KV partition).  The CTA streams its slice of
// the paged K/V ONCE for the whole GQA group (the reference re-streams it per
// q head, pagedattention.metal:957-960): the H_q/H_kv query heads of the group
// are the M rows of an m16n8k16 MMA, 16-token KV tiles are the N (QK^T) / K
// (PV) dimension.  Each of the 4 warps owns every 4th tile of the partition and
// runs its own cp.async ring (16-byte coalesced row segments, zero-filled
// outside the row's [lo, hi) range, XOR-swizzled for conflict-free ldmatrix),
// keeps an online-softmax state in the log2 domain, and the warps are merged
// through shared memory at the end.  Partials go to the split-KV workspace
// (fp32) or, single pass, straight to `out` with the sink fold and the
// 1/(l + 1e-6) normalisation of pagedattention.metal:1318-1328,1383.
//
// HBM-bound: 2 * L * D * esize bytes per (row, kv head); the MMA work
// (4*L*16*D flop) is <2% of the tensor pipe at roofline.
//
// Window mode (WIN; reference pagedattention.metal:1396-1914, host paged_ops.cpp:468-476,508-515): with a
// `window_seqlen_q` hint (spec-decode verification, every segment a K+1-row window) one CTA owns
// floor(16 / G) consecutive query rows of ONE sequence -- they fill the MMA rows the GQA group leaves empty -- and
// streams the KV once for all of them.  Each MMA row keeps its own [lo, hi) range (causal staircase, window start,
// partition clip), tiles are dealt to warps by ABSOLUTE tile index and the split-KV plan is keyed on the row count,
// so every row's arithmetic is the one the expanded (one row per CTA) dispatch does: the two are bitwise equal
// (reference tests/test_spec_window_parity.py).  Tiles on which the rows' masks differ do P.V one query row at a
// time against a V fragment zeroed outside that row's range, so a non-finite V at a position only later rows may see
// cannot reach earlier rows through 0 * inf (test_windowed_skips_masked_inf_v).
//
// KEEP: first positions kept beside a window (WIDE, per-row mode); the tiles that hold them precede the window's, see RowInfo.
//
// DK / DV: compile-time widths of the products over keys and values.  WIDE forms take any size up to that, the columns past
// it zero-filled (a run-time width, whose every step is a branch, ran 1.6 times slower).  WIDE: the softmax weights enter P.V
// as two terms of the operand type; with PACK (at most 8 heads a group) the second terms are the MMA rows the group leaves
// empty, so they cost no product.
#pragma once

#include "paged_attention.cuh"

#include <type_traits>

namespace b200 {

constexpr int kDecodeWarps = 4;
constexpr int kTileTokens = 16;

template <typename T>
struct Mma;
template <>
struct Mma<__nv_bfloat16> {
  __device__ static __forceinline__ void run(float (&c)[4], const uint32_t (&a)[4], uint32_t b0,
                                             uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
        "{%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
  }
  __device__ static __forceinline__ uint32_t pack(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
  }
  __device__ static __forceinline__ uint32_t rest(float lo, float hi, uint32_t packed) {
    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&packed));
    return pack(lo - v.x, hi - v.y);
  }
};
template <>
struct Mma<__half> {
  __device__ static __forceinline__ void run(float (&c)[4], const uint32_t (&a)[4], uint32_t b0,
                                             uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
        "{%8,%9}, {%0,%1,%2,%3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
  }
  __device__ static __forceinline__ uint32_t pack(float lo, float hi) {
    __half2 v = __floats2half2_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
  }
  __device__ static __forceinline__ uint32_t rest(float lo, float hi, uint32_t packed) {
    const float2 v = __half22float2(*reinterpret_cast<const __half2*>(&packed));
    return pack(lo - v.x, hi - v.y);
  }
};

__device__ __forceinline__ void cp_async_16(uint32_t dst, const void* src, int src_bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src),
               "r"(src_bytes)
               : "memory");
}
__device__ __forceinline__ void cp_async_commit() {
  asm volatile("cp.async.commit_group;" ::: "memory");
}
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t& r0, uint32_t& r1, uint32_t& r2,
                                            uint32_t& r3, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t& r0, uint32_t& r1, uint32_t& r2,
                                                  uint32_t& r3, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}

struct DecodeParams {
  void* out;
  const void* query;
  const uint8_t* key_cache;
  const uint8_t* value_cache;
  const int32_t* block_tables;
  const int32_t* seq_lens;
  const int32_t* cu_seqlens_q;
  const float* sinks;
  const float* slopes;  // distance bias: wide, per-row forms only
  int num_seqs, num_q_heads, num_kv_heads, group;
  int block_shift, max_blocks_per_seq, sliding_window, keep_first;
  int64_t q_stride, out_stride;
  uint32_t block_stride16, token_stride16;      // cache strides in 16-byte units
  uint32_t v_block_stride16, v_token_stride16;
  int64_t head_stride_bytes, v_head_stride_bytes;
  int head_dim, value_dim;
  int64_t num_blocks;
  float scale, softcap;
  SplitWorkspace ws;
  int partitioned;
  int win_rows, win_subs;  // window mode: query rows per CTA, CTAs per sequence
};

__host__ __device__ constexpr int decode_ctas_per_sm(int dk, int dv) { return dk >= 128 || dv >= 128 ? 2 : 3; }
__host__ __device__ constexpr int decode_row_bytes(int d) { return (d + 63) / 64 * 128; }  // whole swizzle lines
__host__ __device__ constexpr int decode_tile_bytes(int dk, int dv) {
  return kTileTokens * (decode_row_bytes(dk) + decode_row_bytes(dv));
}
// Tiles a warp of the WIDE forms: what leaves room for the CTAs an SM has registers for, 2 to 4.
constexpr int decode_wide_stages(int dk, int dv) {
  const int fit = (225 * 1024 / decode_ctas_per_sm(dk, dv) - 1024) / (kDecodeWarps * decode_tile_bytes(dk, dv));
  return fit < 2 ? 2 : fit > 4 ? 4 : fit;
}

template <typename T, int DK, int DV, int STAGES, bool WIN, bool WIDE, bool PACK, bool KEEP>
__global__ void __launch_bounds__(kDecodeWarps * 32, decode_ctas_per_sm(DK, DV))
paged_decode_mma_kernel(const DecodeParams p) {
  pdl_trigger();
  pdl_wait();
  constexpr int K_BYTES = decode_row_bytes(DK), V_BYTES = decode_row_bytes(DV);
  constexpr int TILE_BYTES = kTileTokens * K_BYTES;
  constexpr int STAGE_BYTES = decode_tile_bytes(DK, DV);  // K tile then V tile
  constexpr int KSTEPS = DK / 16, VSTEPS = DV / 16;
  static_assert(STAGES * STAGE_BYTES >= 16 * DV * 4, "merge buffer must fit in the ring");
  const int dk = WIDE ? p.head_dim : DK, dv = WIDE ? p.value_dim : DV;
  static_assert(WIDE || DK == DV, "keys and values of different sizes take the wide forms");
  static_assert(!KEEP || (WIDE && !WIN), "kept first positions come with the wide, per-row forms");

  extern __shared__ __align__(128) uint8_t smem_raw[];
  __shared__ float sm_m[kDecodeWarps][16];
  __shared__ float sm_l[kDecodeWarps][16];

  const int kvh = blockIdx.x, part = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, tq = lane & 3;
  const int G = p.group;

  // ---- the CTA's query rows: one (t0), or in window mode nrows consecutive rows of sequence s ----
  int s, t0, nrows, eff0;  // eff0 = KV positions row t0 may see (pagedattention.metal:913); row t0+i sees eff0+i
  RowInfo ri{};
  if constexpr (WIN) {
    s = blockIdx.y / p.win_subs;
    const int r0 = (blockIdx.y - s * p.win_subs) * p.win_rows;
    const int q_start = p.cu_seqlens_q[s];
    const int q_len = p.cu_seqlens_q[s + 1] - q_start;
    if (r0 >= q_len) return;  // shorter segment than the hint: nothing in this sub-window
    nrows = min(p.win_rows, q_len - r0);
    t0 = q_start + r0;
    eff0 = p.seq_lens[s] - q_len + r0 + 1;
  } else {
    t0 = blockIdx.y;
    ri = row_info(p.cu_seqlens_q, p.seq_lens, p.num_seqs, t0, p.sliding_window, p.keep_first, p.ws.skip_qlen);
    s = ri.seq;
    nrows = 1;
    eff0 = ri.eff;
    if (eff0 <= 0) return;  // :917-920
  }
  // KV range [lo, hi) of row t0+qi inside this CTA's partition.  0: the row does not exist (never written),
  // 1: its partition is empty (:922-926), 2: live.
  auto row_range = [&](int qi, int& lo, int& hi) -> int {
    lo = hi = 0;
    const int eff = eff0 + qi;
    if (qi >= nrows || eff <= 0) return 0;
    int beg = 0, base = 0, end = eff;
    if (p.sliding_window >= 0) {  // window: :1129-1133; partitions start at the window's first tile (RowInfo)
      beg = max(0, eff - p.sliding_window);
      base = beg & ~15;
    }
    if (p.partitioned) {
      const int pstart = base + part * p.ws.partition_size;
      if (pstart >= eff) return 1;
      beg = max(beg, pstart);
      end = min(end, pstart + p.ws.partition_size);
    }
    lo = beg;
    hi = max(end, beg);
    return 2;
  };
  // union of the rows' ranges (what is streamed) and their intersection (where no row masks anything)
  int beg, end, ulo = 0, uhi = 0x7fffffff;
  if constexpr (KEEP) {  // two stretches: the range counts tokens without the gap between them
    beg = p.partitioned ? part * p.ws.partition_size : 0;
    end = ri.span();
    if (beg >= end) return;
    if (p.partitioned) end = min(end, beg + p.ws.partition_size);
  } else {
    int umin = 0x7fffffff, umax = 0, live = 0;
    for (int qi = 0; qi < nrows; ++qi) {
      int lo, hi;
      const int st = row_range(qi, lo, hi);
      if (st == 0) continue;
      live |= st == 2;
      if (hi > lo) {
        umin = min(umin, lo);
        umax = max(umax, hi);
      }
      ulo = max(ulo, lo);
      uhi = min(uhi, hi);
    }
    if (!live) return;
    beg = umax > umin ? umin : 0;
    end = umax > umin ? umax : 0;
  }
  const int first_tile = beg >> 4;
  const int n_tiles = end > beg ? ((end - 1) >> 4) - first_tile + 1 : 0;

  // ---- this thread's two MMA rows (g and g+8): query row, head within the group, KV range ----
  int qi0 = 0, qi1 = 0, hl0 = g, hl1 = g + 8;
  if constexpr (WIN) {
    qi0 = g / G;
    hl0 = g - qi0 * G;
    qi1 = (g + 8) / G;
    hl1 = g + 8 - qi1 * G;
  }
  const bool rv0 = WIN ? qi0 < nrows : g < G;
  const bool rv1 = PACK ? false : WIN ? qi1 < nrows : g + 8 < G;
  int lo0 = beg, hi0 = end, lo1 = beg, hi1 = end;
  if constexpr (WIN) {
    row_range(rv0 ? qi0 : nrows, lo0, hi0);
    row_range(rv1 ? qi1 : nrows, lo1, hi1);
  }

  // ---- Q fragments (rows = heads of the GQA group [x query rows], zero beyond) ------------
  uint32_t qf[KSTEPS][4];
  {
    const T* q0 = reinterpret_cast<const T*>(p.query) + (int64_t)(t0 + qi0) * p.q_stride +
                  ((int64_t)kvh * G + hl0) * dk;
    const T* q1 = reinterpret_cast<const T*>(p.query) + (int64_t)(t0 + qi1) * p.q_stride +
                  ((int64_t)kvh * G + hl1) * dk;
#pragma unroll
    for (int ks = 0; ks < KSTEPS; ++ks) {
      const int c = ks * 16 + 2 * tq;
      const bool in0 = c < dk, in1 = c + 8 < dk;  // head sizes are whole 8-element units
      qf[ks][0] = rv0 && in0 ? *reinterpret_cast<const uint32_t*>(q0 + c) : 0u;
      qf[ks][1] = rv1 && in0 ? *reinterpret_cast<const uint32_t*>(q1 + c) : 0u;
      qf[ks][2] = rv0 && in1 ? *reinterpret_cast<const uint32_t*>(q0 + c + 8) : 0u;
      qf[ks][3] = rv1 && in1 ? *reinterpret_cast<const uint32_t*>(q1 + c + 8) : 0u;
    }
  }

  const uint32_t warp_smem =
      (uint32_t)__cvta_generic_to_shared(smem_raw) + warp * (STAGES * STAGE_BYTES);
  const int32_t* table = p.block_tables + (int64_t)s * p.max_blocks_per_seq;
  const int block_mask = (1 << p.block_shift) - 1;
  const uint8_t* kbase = p.key_cache + (int64_t)kvh * p.head_stride_bytes;
  const uint8_t* vbase = p.value_cache + (int64_t)kvh * p.v_head_stride_bytes;

  auto issue_tile = [&](int j, int stage) {
    if (j < n_tiles) {
      const int at = (first_tile + j) * kTileTokens + (lane & 15);
      const int tok = KEEP ? ri.token_at(at) : at;
      int page = tok >> p.block_shift;
      page = min(page, p.max_blocks_per_seq - 1);
      int64_t blk = table[page];
      if (blk < 0 || blk >= p.num_blocks) blk = 0;
      uint32_t koff = (uint32_t)blk * p.block_stride16 + (uint32_t)(tok & block_mask) * p.token_stride16;
      uint32_t voff = (uint32_t)blk * p.v_block_stride16 + (uint32_t)(tok & block_mask) * p.v_token_stride16;
      // zero-fill rows outside the range
      if (at < beg || at >= end || (KEEP && tok < ri.beg && tok >= p.keep_first)) koff = voff = 0xFFFFFFFFu;
      const uint32_t sbase = warp_smem + stage * STAGE_BYTES;
      if constexpr (!WIDE) {  // one layout for both: one row lookup serves K and V
        constexpr int CHUNKS = DK / 8;       // 16-byte chunks per row
        constexpr int ROWS = 32 / CHUNKS;    // rows one warp-wide cp.async covers
        const int c = lane % CHUNKS;
#pragma unroll
        for (int i = 0; i < kTileTokens / ROWS; ++i) {
          const int r = i * ROWS + lane / CHUNKS;
          const uint32_t ro = __shfl_sync(0xffffffffu, koff, r);
          const bool ok = ro != 0xFFFFFFFFu;
          const int64_t goff = (int64_t)(ok ? ro : 0u) * 16 + c * 16;
          const uint32_t dst = sbase + r * K_BYTES + ((c ^ (r & 7)) << 4);
          cp_async_16(dst, kbase + goff, ok ? 16 : 0);
          cp_async_16(dst + TILE_BYTES, vbase + goff, ok ? 16 : 0);
        }
      } else {
        auto copy = [&](auto width, const uint8_t* base, uint32_t off, uint32_t tile, int dim) {
          constexpr int UNITS = decltype(width)::value / 8, PITCH = decode_row_bytes(decltype(width)::value);
#pragma unroll
          for (int i = 0; i < UNITS / 2; ++i) {
            const int at = i * 32 + lane, row = at / UNITS, c = at % UNITS;
            const uint32_t ro = __shfl_sync(0xffffffffu, off, row);
            const bool ok = ro != 0xFFFFFFFFu && c * 8 < dim;
            cp_async_16(tile + row * PITCH + ((c ^ (row & 7)) << 4), base + (int64_t)(ok ? ro + c : 0u) * 16, ok ? 16 : 0);
          }
        };
        copy(std::integral_constant<int, DK>(), kbase, koff, sbase, dk);
        copy(std::integral_constant<int, DV>(), vbase, voff, sbase + TILE_BYTES, dv);
      }
    }
    cp_async_commit();
  };

  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;

  float slope0 = 0.f, slope1 = 0.f;  // log2 units a token
  if (WIDE && !WIN && p.slopes != nullptr) {
    if (rv0) slope0 = p.slopes[kvh * G + hl0] * kLog2e;
    if (rv1) slope1 = p.slopes[kvh * G + hl1] * kLog2e;
  }
  const float sc_mul = p.softcap > 0.f ? p.scale : p.scale * kLog2e;

  // tiles are dealt to warps by absolute index (tile & 3 == warp), so a row's tile -> warp map does not depend on
  // where the CTA's range starts
  const int j0 = (warp - first_tile) & (kDecodeWarps - 1);
#pragma unroll
  for (int st = 0; st < STAGES - 1; ++st) issue_tile(j0 + st * kDecodeWarps, st);

  int stage = 0;
  for (int j = j0; j < n_tiles; j += kDecodeWarps) {
    cp_async_wait<STAGES - 2>();
    __syncwarp();
    {
      int nst = stage + STAGES - 1;
      if (nst >= STAGES) nst -= STAGES;
      issue_tile(j + (STAGES - 1) * kDecodeWarps, nst);
    }
    const uint32_t kt = warp_smem + stage * STAGE_BYTES;
    const uint32_t vt = kt + TILE_BYTES;

    // ---- S = Q K^T : 16 (heads) x 16 (tokens) ---------------------------------
    float sacc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    {
      const int mj = lane >> 3, r = lane & 7;
      const int trow = (mj >> 1) * 8 + r;
#pragma unroll
      for (int ks = 0; ks < KSTEPS; ++ks) {
        const int chunk = ks * 2 + (mj & 1);
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(b0, b1, b2, b3, kt + trow * K_BYTES + ((chunk ^ r) << 4));
        Mma<T>::run(sacc[0], qf[ks], b0, b1);
        Mma<T>::run(sacc[1], qf[ks], b2, b3);
      }
    }
    // ---- scale, softcap, log2 domain, range mask -------------------------------
    const int tok0 = (first_tile + j) * kTileTokens + 2 * tq;
    const int moved = KEEP && first_tile + j >= ri.kept ? ri.gap : 0;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float v = sacc[nt][e] * sc_mul;
        if (p.softcap > 0.f) v = tanhf(v / p.softcap) * p.softcap * kLog2e;  // :1120-1122,1138
        const int tok = tok0 + nt * 8 + (e & 1);
        if (WIDE && !WIN) v = fmaf(e < 2 ? slope0 : slope1, (float)(tok + moved - (eff0 - 1)), v);
        bool in = e < 2 ? (tok >= lo0 && tok < hi0) : (tok >= lo1 && tok < hi1);
        if (KEEP) in = in && (tok + moved >= ri.beg || tok + moved < p.keep_first);
        sacc[nt][e] = in ? v : -INFINITY;
      }
    }
    float mx0 = fmaxf(fmaxf(sacc[0][0], sacc[0][1]), fmaxf(sacc[1][0], sacc[1][1]));
    float mx1 = PACK ? 0.f : fmaxf(fmaxf(sacc[0][2], sacc[0][3]), fmaxf(sacc[1][2], sacc[1][3]));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    if (!PACK) {
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
      mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    }
    const float mn0 = fmaxf(m0, mx0), mn1 = fmaxf(m1, mx1);
    const float mu0 = mn0 == -INFINITY ? 0.f : mn0;  // all masked so far: clamp (:1169-1176)
    const float mu1 = mn1 == -INFINITY ? 0.f : mn1;
    const float c0 = exp2f(m0 - mu0), c1 = PACK ? c0 : exp2f(m1 - mu1);
    m0 = mn0;
    m1 = mn1;
    float ps0 = 0.f, ps1 = 0.f;
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      sacc[nt][0] = exp2f(sacc[nt][0] - mu0);
      sacc[nt][1] = exp2f(sacc[nt][1] - mu0);
      ps0 += sacc[nt][0] + sacc[nt][1];
      if (!PACK) {
        sacc[nt][2] = exp2f(sacc[nt][2] - mu1);
        sacc[nt][3] = exp2f(sacc[nt][3] - mu1);
        ps1 += sacc[nt][2] + sacc[nt][3];
      }
    }
    l0 = l0 * c0 + ps0;
    l1 = l1 * c1 + ps1;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) {
      o[i][0] *= c0;
      o[i][1] *= c0;
      o[i][2] *= c1;
      o[i][3] *= c1;
    }
    // ---- O += P V ---------------------------------------------------------------
    uint32_t pa[4];
    pa[0] = Mma<T>::pack(sacc[0][0], sacc[0][1]);
    pa[1] = PACK ? Mma<T>::rest(sacc[0][0], sacc[0][1], pa[0]) : Mma<T>::pack(sacc[0][2], sacc[0][3]);
    pa[2] = Mma<T>::pack(sacc[1][0], sacc[1][1]);
    pa[3] = PACK ? Mma<T>::rest(sacc[1][0], sacc[1][1], pa[2]) : Mma<T>::pack(sacc[1][2], sacc[1][3]);
    uint32_t pl[4];  // what the operand type leaves of the weights
    if (WIDE && !PACK) {
      pl[0] = Mma<T>::rest(sacc[0][0], sacc[0][1], pa[0]);
      pl[1] = Mma<T>::rest(sacc[0][2], sacc[0][3], pa[1]);
      pl[2] = Mma<T>::rest(sacc[1][0], sacc[1][1], pa[2]);
      pl[3] = Mma<T>::rest(sacc[1][2], sacc[1][3], pa[3]);
    }
    const int tile_beg = (first_tile + j) * kTileTokens;
    // every streamed token of this tile is inside every row's range?  (tokens outside [beg, end) are zero-filled)
    const bool uniform = !WIN || (max(tile_beg, beg) >= ulo && min(tile_beg + kTileTokens, end) <= uhi);
    if (uniform) {
      const int mj = lane >> 3, r = lane & 7;
      const int trow = (mj & 1) * 8 + r;
#pragma unroll
      for (int n2 = 0; n2 < VSTEPS; ++n2) {
        const int chunk = n2 * 2 + (mj >> 1);
        uint32_t v0, v1, v2, v3;
        ldmatrix_x4_trans(v0, v1, v2, v3, vt + trow * V_BYTES + ((chunk ^ r) << 4));
        Mma<T>::run(o[2 * n2], pa, v0, v1);
        Mma<T>::run(o[2 * n2 + 1], pa, v2, v3);
        if (WIDE && !PACK) {
          Mma<T>::run(o[2 * n2], pl, v0, v1);
          Mma<T>::run(o[2 * n2 + 1], pl, v2, v3);
        }
      }
    } else {
      // the rows' masks differ on this tile: one query row at a time, V zeroed outside that row's range -- what the
      // expanded dispatch's zero-filled load gives that row; the other rows keep their accumulators
      const int mj = lane >> 3, r = lane & 7;
      const int trow = (mj & 1) * 8 + r;
      const int tk = tile_beg + 2 * tq;  // this lane's B-fragment tokens: tk, tk+1 (b0) and tk+8, tk+9 (b1)
      for (int qi = 0; qi < nrows; ++qi) {
        int lo, hi;
        row_range(qi, lo, hi);
        const uint32_t m01 = ((tk >= lo && tk < hi) ? 0x0000FFFFu : 0u) | ((tk + 1 >= lo && tk + 1 < hi) ? 0xFFFF0000u : 0u);
        const uint32_t m89 = ((tk + 8 >= lo && tk + 8 < hi) ? 0x0000FFFFu : 0u) | ((tk + 9 >= lo && tk + 9 < hi) ? 0xFFFF0000u : 0u);
        // only query row qi's MMA rows take this pass's result: a zero P row times a non-finite V is NaN, not 0
        const bool t0_ = rv0 && qi0 == qi, t1_ = rv1 && qi1 == qi;
        uint32_t pq[4];
        pq[0] = t0_ ? pa[0] : 0u;
        pq[1] = t1_ ? pa[1] : 0u;
        pq[2] = t0_ ? pa[2] : 0u;
        pq[3] = t1_ ? pa[3] : 0u;
#pragma unroll
        for (int n2 = 0; n2 < VSTEPS; ++n2) {
            const int chunk = n2 * 2 + (mj >> 1);
          uint32_t v0, v1, v2, v3;
          ldmatrix_x4_trans(v0, v1, v2, v3, vt + trow * V_BYTES + ((chunk ^ r) << 4));
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            float (&oo)[4] = o[2 * n2 + h];
            float d[4] = {oo[0], oo[1], oo[2], oo[3]};
            Mma<T>::run(d, pq, (h ? v2 : v0) & m01, (h ? v3 : v1) & m89);
            if (t0_) {
              oo[0] = d[0];
              oo[1] = d[1];
            }
            if (t1_) {
              oo[2] = d[2];
              oo[3] = d[3];
            }
          }
        }
      }
    }
    if (++stage == STAGES) stage = 0;
  }
  cp_async_wait<0>();
  __syncwarp();

  if (PACK)
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) {
      o[i][0] += o[i][2];
      o[i][1] += o[i][3];
    }
  // ---- per-warp state -> shared memory, then merge the 4 warps -------------------
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1);
  l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  float* so = reinterpret_cast<float*>(smem_raw + warp * (STAGES * STAGE_BYTES));
  if (tq == 0) {
    sm_m[warp][g] = m0;
    sm_l[warp][g] = l0;
    sm_m[warp][g + 8] = m1;
    sm_l[warp][g + 8] = l1;
  }
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) {
    if (rv0) *reinterpret_cast<float2*>(so + g * DV + i * 8 + 2 * tq) = make_float2(o[i][0], o[i][1]);
    if (rv1)
      *reinterpret_cast<float2*>(so + (g + 8) * DV + i * 8 + 2 * tq) = make_float2(o[i][2], o[i][3]);
  }
  __syncthreads();

  for (int idx = threadIdx.x; idx < nrows * G * dv; idx += blockDim.x) {
    const int row = idx / dv, d = idx - row * dv;  // MMA row = query row * G + head within the group
    const int qi = WIN ? row / G : 0;
    const int t = t0 + qi;
    if (WIN && eff0 + qi <= 0) continue;  // :917-920
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < kDecodeWarps; ++w) M = fmaxf(M, sm_m[w][row]);
    float L = 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < kDecodeWarps; ++w) {
      const float mw = sm_m[w][row];
      if (mw != -INFINITY) {  // skip warps that saw nothing (:1288-1289)
        const float wgt = exp2f(mw - M);
        L += sm_l[w][row] * wgt;
        const float* sw =
            reinterpret_cast<const float*>(smem_raw + w * (STAGES * STAGE_BYTES));
        acc += sw[row * DV + d] * wgt;
      }
    }
    const int h = kvh * G + (row - qi * G);
    if (p.partitioned) {
      const int64_t prow = ((int64_t)t * p.num_q_heads + h) * p.ws.num_partitions + part;
      p.ws.tmp_out[prow * dv + d] = acc;
      if (d == 0) {
        p.ws.max_l2[prow] = M;
        p.ws.exp_sum[prow] = L;
      }
    } else {
      if (M == -INFINITY) M = 0.f;
      float c = 1.f;
      if (p.sinks != nullptr) {  // :1318-1328
        const float sk = p.sinks[h] * kLog2e;
        const float M2 = fmaxf(M, sk);
        c = exp2f(M - M2);
        L = L * c + exp2f(sk - M2);
      }
      T* op = reinterpret_cast<T*>(p.out) + (int64_t)t * p.out_stride + (int64_t)h * dv;
      store_out<T>(op, d, acc * c / (L + p.ws.denom_eps), p.ws.out_f16);  // :1383
    }
  }
}

template <typename T, int DK, int DV, int STAGES, bool WIN, bool WIDE, bool PACK = false, bool KEEP = false>
int launch_decode_form(const DecodeParams& p, dim3 grid, cudaStream_t st) {
  constexpr int smem = kDecodeWarps * STAGES * decode_tile_bytes(DK, DV);
  static bool configured_dev[16] = {false};  // cudaFuncSetAttribute is per device
  int dev = 0;
  B200_CUDA_OK(cudaGetDevice(&dev));
  if (!configured_dev[dev & 15]) {
    B200_CUDA_OK(cudaFuncSetAttribute(paged_decode_mma_kernel<T, DK, DV, STAGES, WIN, WIDE, PACK, KEEP>,
                                      cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    configured_dev[dev & 15] = true;
  }
  launch_pdl(paged_decode_mma_kernel<T, DK, DV, STAGES, WIN, WIDE, PACK, KEEP>, grid, dim3(kDecodeWarps * 32), smem, st, p);
  return check_launch("paged_decode_mma_kernel");
}

// The WIDE forms by the smallest widths that hold the head sizes (paged_attention_decode_wide.cuh).
constexpr int decode_key_width(int d) { return d <= 64 ? 64 : d <= 96 ? 96 : d <= 128 ? 128 : 256; }
constexpr int decode_value_width(int d) { return d <= 64 ? 64 : d <= 128 ? 128 : d <= 192 ? 192 : 256; }
int launch_decode_wide(const DecodeParams& p, dim3 grid, cudaStream_t st);         // any group
int launch_decode_wide_packed(const DecodeParams& p, dim3 grid, cudaStream_t st);  // at most 8 heads a group
int launch_decode_kept(const DecodeParams& p, dim3 grid, cudaStream_t st);         // the same with kept first positions
int launch_decode_kept_packed(const DecodeParams& p, dim3 grid, cudaStream_t st);

}  // namespace b200
