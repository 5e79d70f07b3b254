// Latent attention for decode on tcgen05 (bf16), transposed so that the cached rows fill the M side of every product:
//   S^T [keys x rows]  = C Q^T        A = a tile of 64 cached rows (K-major), B = 32 (token, head) rows of queries
//   O^T [dims x rows] += C^T P^T      A = the same tile read MN-major (its latent columns), B = the softmax weights
// so a cached row crosses HBM once and shared memory holds it once for both products, and few heads waste no tensor
// rows.  The weights stay 16 bits wide through the value product: B is [P_hi | P_lo], 64 columns, two accumulators.
//
//   warps 0, 2, 3  TMA: per 64-key tile the pages named by the block table, one box per page and 64-column slice, the
//             slices dealt out to the three warps (a box takes ~50 cycles to issue)
//   warp 1    MMA issuer; S^T of the next tile goes out as soon as its rows have landed, before the value product of
//             this tile if that still waits for its weights
//   warps 4-11 two groups of four (one warp per tensor-memory lane quarter), 16 rows a group.  The quarters that hold
//             keys do the softmax, thread = key: weights against a reference maximum per row that only moves when a
//             score exceeds it by more than 2^8 -- one vote per tile; then all warps rescale O^T.  Private row sums;
//             final division and store by all.
// The S^T product addresses 128 rows of which the tile holds 64; the other half lands in tensor memory nobody reads.
#pragma once

#include "../../include/b200_hybrid_ops.h"
#include "tcgen05.cuh"

namespace b200 {
namespace latent_tc {
using namespace tc;

constexpr int kRows = 32, kKeys = 64, kStages = 2, kThreads = 384;
constexpr int kHalf = kRows / 2, kGroup = 256;  // softmax / correction threads
constexpr int kSliceBytes = kKeys * 128, kQSliceBytes = kRows * 128, kPBytes = kKeys * 128;
constexpr int kMaxSlices = 10;  // 640 columns
constexpr int TM_S = 0, TM_O = 2 * kRows;
constexpr float kRescale = 8.f;  // log2 units

__device__ int g_failed = 0;  // a wait ran out: results of the launch are invalid

struct Params {
  const int32_t* block_tables;
  const int32_t* seq_lens;
  const int32_t* cu;
  void* out;
  float* wo;
  int num_tokens, heads, rank, width, slices, mtiles, block_size, max_blocks, window, max_q_len, splits;
  float scale2;  // scale * log2(e)
};

inline int smem_bytes(int slices) {
  return kStages * slices * kSliceBytes + slices * kQSliceBytes + 2 * kPBytes + 2048 + 1024;
}

__device__ __forceinline__ float ex2f(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float redux_max(float x) {
  float y;
  asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(y) : "f"(x));
  return y;
}

__device__ __forceinline__ bool group_any(bool x) {
  uint32_t y;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.b32 p, %1, 0;\n\t"
      "barrier.cta.red.or.pred q, 1, 256, p;\n\t"
      "selp.u32 %0, 1, 0, q;\n\t}"
      : "=r"(y)
      : "r"((uint32_t)x)
      : "memory");
  return y != 0;
}

__global__ void __launch_bounds__(kThreads, 1)
latent_tc_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap c_map, const Params p) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.y, split = blockIdx.z;
  const int row0 = p.cu[s], len = p.cu[s + 1] - row0, seq_len = p.seq_lens[s];
  const int r_first = blockIdx.x * kRows;
  if (len <= 0 || len > p.max_q_len || r_first >= len * p.heads) return;
  const int nrows = min(kRows, len * p.heads - r_first);
  const int start = seq_len - len;
  const int pos_first = start + r_first / p.heads, pos_last = start + (r_first + nrows - 1) / p.heads;
  const int lo_all = p.window > 0 ? max(0, pos_first - p.window + 1) : 0, hi_all = pos_last + 1;
  const int t0 = lo_all / kKeys, tiles = (hi_all + kKeys - 1) / kKeys - t0;
  const int t_begin = t0 + (int)((int64_t)tiles * split / p.splits), t_end = t0 + (int)((int64_t)tiles * (split + 1) / p.splits);
  const int nt = t_end - t_begin;

  extern __shared__ __align__(1024) uint8_t raw[];
  const uint32_t base = (smem_u32(raw) + 1023u) & ~1023u;
  const uint32_t stage_bytes = p.slices * kSliceBytes;
  const uint32_t sm_c = base, sm_q = sm_c + kStages * stage_bytes, sm_p = sm_q + p.slices * kQSliceBytes;
  const uint32_t sm_bar = sm_p + 2 * kPBytes;
  const uint32_t bar_q = sm_bar, bar_full = sm_bar + 8, bar_s = bar_full + 16, bar_p = bar_s + 16, bar_o = bar_p + 16;
  const uint32_t tmem_ptr = bar_o + 16;
  uint8_t* gen = raw + (base - smem_u32(raw));
  volatile uint32_t* tmem_gen = reinterpret_cast<volatile uint32_t*>(gen + (tmem_ptr - base));
  float* smax = reinterpret_cast<float*>(gen + (sm_bar - base) + 128);  // [2 tile parities][2 warps][32]
  float* ssum = smax + 128;                                              // [2 warps][32]
  float* sref = ssum + 64;                                               // [32] reference maxima at the end
  volatile int* sfail = reinterpret_cast<volatile int*>(sref + 32);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(bar_q, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(bar_full + 8 * i, 1);
      mbar_init(bar_s + 8 * i, 1);
      mbar_init(bar_p + 8 * i, 8);
      mbar_init(bar_o + 8 * i, 1);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    *sfail = 0;
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tmem_ptr), "n"(512) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_gen;

  if (warp == 0 || warp == 2 || warp == 3) {
    // ===== TMA producers =====
    const int lane_of = warp == 0 ? 0 : warp - 1;  // this warp's slices: lane_of, lane_of + 3, ...
    const int32_t* table = p.block_tables + (int64_t)s * p.max_blocks;
    if (warp == 0 && elect_one()) {
      mbar_expect_tx(bar_q, p.slices * kQSliceBytes);
      for (int i = 0; i < p.slices; ++i)
        tma_load_2d(sm_q + i * kQSliceBytes, &q_map, bar_q, i * 64, row0 * p.heads + r_first);
    }
    __syncwarp();
    const int pages = kKeys / p.block_size, page_bytes = p.block_size * 128;
    int issued = 0;
    auto page_of = [&](int t) {  // lane l holds page l; pages past the last visible key read page 0 and are masked
      const int pg = (t_begin + t) * pages + lane;
      return lane < pages && pg < p.max_blocks && pg * p.block_size < hi_all ? table[pg] : 0;
    };
    int next = page_of(0);
    for (int t = 0; t < nt; ++t) {
      const int st = t & 1, page = next;
      if (t + 1 < nt) next = page_of(t + 1);
      if (t >= 2 && !mbar_wait_or_fail(bar_o + 8 * st, ((t - 2) >> 1) & 1)) {
        if (lane == 0) *sfail = 1;
        break;
      }
      if (warp == 0 && elect_one()) mbar_expect_tx(bar_full + 8 * st, stage_bytes);
      __syncwarp();
      for (int g = 0; g < pages; ++g) {
        const int row = __shfl_sync(0xffffffffu, page, g) * p.block_size;
        if (elect_one())
          for (int i = lane_of; i < p.slices; i += 3)
            tma_load_2d(sm_c + st * stage_bytes + i * kSliceBytes + g * page_bytes, &c_map, bar_full + 8 * st, i * 64, row);
        __syncwarp();
      }
      issued = t + 1;
    }
    // whatever happened, the copies in flight land before the CTA's memory goes away
    mbar_wait_or_fail(bar_q, 0);
    for (int t = max(0, issued - 2); t < issued; ++t) mbar_wait_or_fail(bar_full + 8 * (t & 1), (t >> 1) & 1);
  } else if (warp == 1) {
    // ===== MMA issuer =====
    const uint32_t idesc_s = make_idesc(1, 128, kRows);
    const uint32_t idesc_o = make_idesc(1, 128, 2 * kRows) | (1u << 15) | (1u << 16);  // A and B MN-major
    const uint32_t tb = __shfl_sync(0xffffffffu, tmem, 0);
    const int ksteps = (p.width + 15) >> 4, full = ksteps >> 2;
    const uint64_t dq = make_smem_desc(sm_q);
    bool ok = mbar_wait_or_fail(bar_q, 0);
    auto issue_s = [&](int t) {
      const int st = t & 1;
      if (!mbar_wait_or_fail(bar_full + 8 * st, (t >> 1) & 1)) return false;
      tc_fence_after();
      if (elect_one()) {
        // descriptors advance by adding to their address field (16-byte units)
        const uint64_t da = make_smem_desc(sm_c + st * stage_bytes);
        for (int i = 0; i < full; ++i) {
#pragma unroll
          for (int k = 0; k < 4; ++k)
            tc_mma_f16(tb + TM_S + st * kRows, da + i * (kSliceBytes >> 4) + 2 * k, dq + i * (kQSliceBytes >> 4) + 2 * k,
                       idesc_s, (i | k) == 0 ? 0u : 1u);
        }
        for (int k = full * 4; k < ksteps; ++k)
          tc_mma_f16(tb + TM_S + st * kRows, da + full * (kSliceBytes >> 4) + 2 * (k & 3),
                     dq + full * (kQSliceBytes >> 4) + 2 * (k & 3), idesc_s, k == 0 ? 0u : 1u);
        tc_commit(bar_s + 8 * st);
      }
      __syncwarp();
      return true;
    };
    ok = ok && nt > 0 && issue_s(0);
    for (int t = 0; ok && t < nt; ++t) {
      const int st = t & 1;
      bool ahead = t + 1 == nt;  // S^T of the next tile is on its way (or there is none)
      bool ready = false;
      for (uint32_t spins = 0; !ready && ok && spins < (1u << 26); ++spins) {
        if (!ahead && mbar_test(bar_full + 8 * (st ^ 1), ((t + 1) >> 1) & 1)) ok = ahead = issue_s(t + 1);
        ready = mbar_test(bar_p + 8 * st, (t >> 1) & 1);
      }
      if (!(ok = ok && ready)) break;
      // rows past the last visible key are whatever the pool holds; their weights are 0, but 0 * NaN is not
      const int valid = hi_all - (t_begin + t) * kKeys;
      if (valid < kKeys) {
        const int per = 8 * p.slices;
        for (int i = lane; i < (kKeys - valid) * per; i += 32) {
          const int row = valid + i / per, rem = i % per;
          asm volatile("st.shared.v4.u32 [%0], {%1,%1,%1,%1};" ::"r"(sm_c + st * stage_bytes + (rem >> 3) * kSliceBytes +
                                                                     row * 128 + (rem & 7) * 16), "r"(0u) : "memory");
        }
        fence_proxy_async();
        __syncwarp();
      }
      tc_fence_after();
      if (elect_one()) {
        const uint64_t dc = make_smem_desc_mn(sm_c + st * stage_bytes, kSliceBytes, 1024);
        const uint64_t dp = make_smem_desc_mn(sm_p + st * kPBytes, kPBytes, 1024);
        for (int i = 0; i < p.mtiles; ++i) {
#pragma unroll
          for (int k = 0; k < kKeys / 16; ++k)
            tc_mma_f16(tb + TM_O + i * 2 * kRows, dc + 2 * i * (kSliceBytes >> 4) + k * (2048 >> 4), dp + k * (2048 >> 4),
                       idesc_o, (t | k) != 0 ? 1u : 0u);
        }
        tc_commit(bar_o + 8 * st);
      }
      __syncwarp();
      if (!ahead) ok = issue_s(t + 1);
    }
    if (!ok && nt > 0 && lane == 0) *sfail = 1;
  } else if (warp >= 4) {
    // ===== softmax, rescaling =====
    const int q = warp & 3, half = (warp - 4) >> 2, rbase = half * kHalf;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    float ref[kHalf], lsum[kHalf];  // reference maxima (log2 units, the same in all of the group) and private sums
#pragma unroll
    for (int r = 0; r < kHalf; ++r) ref[r] = -INFINITY, lsum[r] = 0.f;
    bool ok = true;
    for (int t = 0; t < nt; ++t) {
      const int st = t & 1;
      float v[kHalf];
      bool over = false;
      if (q < 2) {
        ok = ok && mbar_wait_or_fail(bar_s + 8 * st, (t >> 1) & 1);
        tc_fence_after();
        uint32_t u[16];
        tmem_ld<16>(tmem + lane_addr + TM_S + st * kRows + rbase, u);
        const int key0 = (t_begin + t) * kKeys, key = key0 + q * 32 + lane;
#pragma unroll
        for (int r = 0; r < kHalf; ++r) v[r] = __uint_as_float(u[r]) * p.scale2;
        if (key0 + kKeys > pos_first + 1 || (p.window > 0 && pos_last - key0 >= p.window) || nrows < kRows) {
          int pos = start + (r_first + rbase) / p.heads, left = p.heads - (r_first + rbase) % p.heads;
#pragma unroll
          for (int r = 0; r < kHalf; ++r) {
            if (rbase + r >= nrows || key > pos || (p.window > 0 && pos - key >= p.window)) v[r] = -INFINITY;
            if (--left == 0) ++pos, left = p.heads;
          }
        }
#pragma unroll
        for (int r = 0; r < kHalf; ++r) over |= v[r] > ref[r] + kRescale;
      }
      if (group_any(over)) {
        float* sm = smax + st * 64;
        if (q < 2) {
          float mx = -INFINITY;
#pragma unroll
          for (int r = 0; r < kHalf; ++r) {
            const float rm = redux_max(v[r]);
            if (lane == r) mx = rm;
          }
          if (lane < kHalf) sm[q * 32 + rbase + lane] = mx;
        }
        asm volatile("bar.sync 1, 256;" ::: "memory");
        float alpha[kHalf];
#pragma unroll
        for (int r = 0; r < kHalf; ++r) {
          const float mt = fmaxf(sm[rbase + r], sm[32 + rbase + r]);
          const float mn = mt > ref[r] + kRescale ? mt : ref[r];
          alpha[r] = ref[r] == -INFINITY ? 1.f : ex2f(ref[r] - mn);
          ref[r] = mn;
          lsum[r] *= alpha[r];
        }
        if (t > 0) {
          ok = ok && mbar_wait_or_fail(bar_o + 8 * ((t - 1) & 1), ((t - 1) >> 1) & 1);
          tc_fence_after();
          for (int i = 0; i < 2 * p.mtiles; ++i) {
            uint32_t u[16];
            tmem_ld<16>(tmem + lane_addr + TM_O + i * kRows + rbase, u);
#pragma unroll
            for (int r = 0; r < kHalf; ++r) u[r] = __float_as_uint(__uint_as_float(u[r]) * alpha[r]);
            tmem_st16(tmem + lane_addr + TM_O + i * kRows + rbase, u);
          }
        }
      }
      if (q < 2) {
        if (t >= 2) ok = ok && mbar_wait_or_fail(bar_o + 8 * st, ((t - 2) >> 1) & 1);
        uint32_t hi[8], lo[8];
#pragma unroll
        for (int r = 0; r < kHalf; r += 2) {
          const float p0 = ref[r] == -INFINITY ? 0.f : ex2f(v[r] - ref[r]);
          const float p1 = ref[r + 1] == -INFINITY ? 0.f : ex2f(v[r + 1] - ref[r + 1]);
          lsum[r] += p0;
          lsum[r + 1] += p1;
          const __nv_bfloat162 h = __floats2bfloat162_rn(p0, p1);
          const __nv_bfloat162 l = __floats2bfloat162_rn(p0 - __low2float(h), p1 - __high2float(h));
          hi[r >> 1] = *reinterpret_cast<const uint32_t*>(&h);
          lo[r >> 1] = *reinterpret_cast<const uint32_t*>(&l);
        }
        const int k = q * 32 + lane;
        const uint32_t dst = sm_p + st * kPBytes + k * 128;
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const int ch = half * 2 + c;
          asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};" ::"r"(dst + ((ch ^ (k & 7)) << 4)), "r"(hi[4 * c]),
                       "r"(hi[4 * c + 1]), "r"(hi[4 * c + 2]), "r"(hi[4 * c + 3]) : "memory");
          asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};" ::"r"(dst + (((ch + 4) ^ (k & 7)) << 4)), "r"(lo[4 * c]),
                       "r"(lo[4 * c + 1]), "r"(lo[4 * c + 2]), "r"(lo[4 * c + 3]) : "memory");
        }
        fence_proxy_async();
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_p + 8 * st);
    }  // a warp whose wait ran out keeps its place in the group's barriers and waits for nothing more
    if (nt > 0) ok = ok && mbar_wait_or_fail(bar_o + 8 * ((nt - 1) & 1), ((nt - 1) >> 1) & 1);
    if (!ok && lane == 0) *sfail = 1;
    tc_fence_after();
    if (q < 2) {
#pragma unroll
      for (int r = 0; r < kHalf; ++r) {
        const float x = warp_sum(lsum[r]);
        if (lane == r) ssum[q * 32 + rbase + r] = x;
        if (q == 0 && lane == r) sref[rbase + r] = ref[r];
      }
    }
  }
  __syncthreads();
  if (*sfail) {
    if (threadIdx.x == 0) atomicExch(&g_failed, 1);
  } else if (warp >= 4) {
    const int q = warp & 3, rbase = ((warp - 4) >> 2) * kHalf;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    const size_t all_rows = (size_t)p.num_tokens * p.heads, first = (size_t)row0 * p.heads + r_first;
    if (p.splits > 1 && warp == 4 && lane < nrows) {
      float* wml = p.wo + (size_t)p.splits * all_rows * p.rank;
      wml[2 * (split * all_rows + first + lane)] = sref[lane];
      wml[2 * (split * all_rows + first + lane) + 1] = ssum[lane] + ssum[32 + lane];
    }
    float inv[kHalf];
#pragma unroll
    for (int r = 0; r < kHalf; ++r) inv[r] = p.splits == 1 ? 1.f / (ssum[rbase + r] + ssum[32 + rbase + r]) : 1.f;
    for (int i = 0; i < p.mtiles; ++i) {
      const int dim = i * 128 + q * 32 + lane;
      uint32_t a[16], b[16];
      if (nt > 0) {
        tmem_ld<16>(tmem + lane_addr + TM_O + i * 2 * kRows + rbase, a);
        tmem_ld<16>(tmem + lane_addr + TM_O + i * 2 * kRows + kRows + rbase, b);
      }
#pragma unroll
      for (int r = 0; r < kHalf; ++r) {
        if (rbase + r >= nrows || dim >= p.rank) continue;
        const float x = nt > 0 ? (__uint_as_float(a[r]) + __uint_as_float(b[r])) * inv[r] : 0.f;
        if (p.splits == 1) {
          reinterpret_cast<__nv_bfloat16*>(p.out)[(first + rbase + r) * p.rank + dim] = __float2bfloat16_rn(x);
        } else {
          p.wo[((size_t)split * all_rows + first + rbase + r) * p.rank + dim] = x;
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(512) : "memory");
  }
}

}  // namespace latent_tc
}  // namespace b200
