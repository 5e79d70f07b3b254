// Products of all routed experts (and of a shared one) in one persistent launch on tcgen05, bf16.
//
// Weights fill the M side and tokens the N side, so an expert's weights cross HBM once for up to TOKENS tokens however few
// there are, and a launch serves a decode step as well as a prompt.  Work items are (stretch, 128 or 256 output features,
// tile of TOKENS sorted pairs); a CTA takes every gridDim.x-th one and its producers run ahead across items.
//   gated    (the way in):  two accumulators, gate and up rows of the same 128 features, silu(gate) * up in the epilogue
//   straight (the way out): two accumulators, features f .. f + 127 and f + 128 .. f + 255
//
//   warp 0     TMA producer: weight tiles (straight: also the token tile, consecutive rows of the sorted activations)
//   warp 1     MMA issuer: D_h[128 features x TOKENS] += W_h[128 x 64] X[TOKENS x 64]^T per 64-column step, h = 0, 1
//   warps 2-5  epilogue, thread = feature, stores in pairs; two pairs of accumulators, so the next item's products
//              overlap it
//   warps 6-9  (gated) the token tile: rows gathered by pair with 16-byte asynchronous copies into the swizzled layout
// Products are as wide as the tile has rows, in steps of 16; the columns of rows past a stretch's end go nowhere.
#pragma once

#include "../../include/b200_hybrid_ops.h"
#include "tcgen05.cuh"

#include <type_traits>

namespace b200 {

// The stretch that holds tile `i`: the last one whose running count is not past it (empty ones are stepped over).
__device__ __forceinline__ int find_stretch(const int32_t* tiles, int n, int i) {
  int lo = 0, hi = n;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (tiles[mid] <= i) lo = mid; else hi = mid;
  }
  return lo;
}

namespace experts_tc {
using namespace tc;

constexpr int kSlab = 64;                 // columns of K per stage
constexpr int kHalfBytes = 128 * 128;     // 128 weight rows x 64 columns
constexpr int kGatherLag = 3;             // stages of gathered rows in flight

__device__ int g_failed = 0;  // a wait ran out or the plan was not sound: results of the launch are invalid

struct Params {
  const int32_t* pairs;
  const int32_t* first;
  const int32_t* tiles;
  const __nv_bfloat16* x;  // gated: rows to gather
  __nv_bfloat16* out;
  __nv_bfloat16* shared_out;
  int64_t x_stride, out_stride, shared_out_stride;
  int rows, experts, top, n_out, k, shared_n_out, shared_k, shared_tiles, max_tiles;
};

template <int TOKENS>
struct Shape {
  static constexpr int X_BYTES = TOKENS * 128, STAGE_BYTES = 2 * kHalfBytes + X_BYTES;
  static constexpr int STAGES = TOKENS <= 64 ? 5 : 4;
  static constexpr int TMEM_COLS = 4 * TOKENS;            // two accumulator pairs
  static constexpr int BOX = TOKENS < 64 ? TOKENS : 64;   // rows of a token tile per copy
};
inline int smem_bytes(int stages, int stage_bytes, int experts) { return stages * stage_bytes + 1024 + 256 + 8 * (experts + 1); }

struct Item {
  bool shared;
  int feature, row0, nrows, w_row, k, n_out;
};

template <int TOKENS, bool GATED>
struct Work {
  static constexpr int FEATURES = GATED ? 128 : 256;
  int ft, fts, shared_items, total;
  __device__ __forceinline__ Work(const Params& p, const int* tiles) {
    ft = (p.n_out + FEATURES - 1) / FEATURES;
    fts = p.shared_tiles > 0 ? (p.shared_n_out + FEATURES - 1) / FEATURES : 0;
    shared_items = fts * p.shared_tiles;
    total = shared_items + tiles[p.experts] * ft;
  }
  __device__ __forceinline__ Item at(const Params& p, const int* tiles, const int* first, int i) const {
    Item w;
    int tile;
    w.shared = i < shared_items;
    if (w.shared) {
      const int f = i / p.shared_tiles;
      tile = i - f * p.shared_tiles;
      w.feature = f * FEATURES;
      w.row0 = tile * TOKENS;
      w.nrows = min(TOKENS, p.rows - w.row0);
      w.w_row = 0;
      w.k = p.shared_k;
      w.n_out = p.shared_n_out;
    } else {
      i -= shared_items;
      const int e = find_stretch(tiles, p.experts, i / ft), n = tiles[e + 1] - tiles[e];
      const int local = i - tiles[e] * ft, f = local / n;
      tile = local - f * n;
      w.feature = f * FEATURES;
      w.row0 = first[e] + tile * TOKENS;
      w.nrows = min(TOKENS, first[e + 1] - w.row0);
      w.w_row = e * p.n_out * (GATED ? 2 : 1);
      w.k = p.k;
      w.n_out = p.n_out;
    }
    return w;
  }
};

// Lane l holds columns c0 and c1 of feature l: an even lane gets (l, l + 1) of c0, an odd one (l - 1, l) of c1.
__device__ __forceinline__ uint32_t swap_pack(uint32_t c0, uint32_t c1) {
  const bool odd = threadIdx.x & 1;
  const uint32_t other = __shfl_xor_sync(0xffffffffu, odd ? c0 : c1, 1);
  const __nv_bfloat162 v = __floats2bfloat162_rn(__uint_as_float(odd ? other : c0), __uint_as_float(odd ? c1 : other));
  return *reinterpret_cast<const uint32_t*>(&v);
}

template <int TOKENS, bool GATED>
__global__ void __launch_bounds__(GATED ? 320 : 192, 1)
expert_product_tc_kernel(const __grid_constant__ CUtensorMap w_map, const __grid_constant__ CUtensorMap x_map,
                         const __grid_constant__ CUtensorMap sw_map, const __grid_constant__ CUtensorMap sx_map, const Params p) {
  using SH = Shape<TOKENS>;
  constexpr int STAGES = SH::STAGES;
  extern __shared__ __align__(1024) uint8_t raw[];
  const uint32_t base = (smem_u32(raw) + 1023u) & ~1023u;
  const uint32_t sm_bar = base + STAGES * SH::STAGE_BYTES;
  const uint32_t bar_full = sm_bar, bar_empty = bar_full + 8 * STAGES, bar_acc = bar_empty + 8 * STAGES, bar_free = bar_acc + 16;
  const uint32_t tmem_ptr = bar_free + 16;
  uint8_t* gen = raw + (base - smem_u32(raw)) + STAGES * SH::STAGE_BYTES;
  volatile uint32_t* tmem_gen = reinterpret_cast<volatile uint32_t*>(gen + (tmem_ptr - sm_bar));
  volatile int* sfail = reinterpret_cast<volatile int*>(gen + (tmem_ptr - sm_bar) + 4);
  int* tiles = reinterpret_cast<int*>(gen + 256);
  int* first = tiles + p.experts + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_trigger();
  if (threadIdx.x == 0) {
    for (int i = 0; i < STAGES; ++i) {
      mbar_init(bar_full + 8 * i, GATED ? 5 : 1);
      mbar_init(bar_empty + 8 * i, 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(bar_acc + 8 * i, 1);
      mbar_init(bar_free + 8 * i, 4);
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    *sfail = 0;
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(tmem_ptr), "n"(SH::TMEM_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  pdl_wait();
  // The plan is checked on the way in: running counts that fit together, so that whatever they hold, every row below is
  // a row of the operands.
  const int pairs_total = p.rows * p.top;
  for (int i = threadIdx.x; i <= p.experts; i += blockDim.x) {
    const int t = p.tiles[i], f = p.first[i];
    tiles[i] = t;
    first[i] = f;
    const int tn = i < p.experts ? p.tiles[i + 1] : t, fn = i < p.experts ? p.first[i + 1] : pairs_total;
    if (t < 0 || f < 0 || t > p.max_tiles || f > pairs_total || (i < p.experts && (fn < f || tn - t != (fn - f + TOKENS - 1) / TOKENS)))
      *sfail = 1;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_gen;
  const bool sound = *sfail == 0;
  __syncthreads();
  Work<TOKENS, GATED> work(p, tiles);
  if (!sound) work.total = 0;

  auto pair_at = [&](int i) { return (int)min((uint32_t)p.pairs[i], (uint32_t)pairs_total - 1); };

  if (warp == 0) {
    // ===== TMA producer =====
    int n = 0;  // stages issued
    bool ok = true;
    for (int i = blockIdx.x; ok && i < work.total; i += gridDim.x) {
      const Item w = work.at(p, tiles, first, i);
      const int slabs = (w.k + kSlab - 1) / kSlab;
      const bool both = GATED || w.feature + 128 < w.n_out;
      const int r0 = w.w_row + w.feature, r1 = r0 + (GATED ? w.n_out : 128);
      const CUtensorMap* wm = w.shared ? &sw_map : &w_map;
      const CUtensorMap* xm = w.shared ? &sx_map : &x_map;
      for (int s = 0; s < slabs; ++s, ++n) {
        const int st = n % STAGES;
        const uint32_t dst = base + st * SH::STAGE_BYTES, bar = bar_full + 8 * st;
        if (!(ok = mbar_wait_or_fail(bar_empty + 8 * st, ((n / STAGES) & 1) ^ 1))) break;
        if (elect_one()) {
          const int boxes = GATED ? 0 : (w.nrows + SH::BOX - 1) / SH::BOX;
          mbar_expect_tx(bar, (both ? 2 : 1) * kHalfBytes + boxes * SH::BOX * 128);
          tma_load_2d(dst, wm, bar, s * kSlab, r0);
          if (both) tma_load_2d(dst + kHalfBytes, wm, bar, s * kSlab, r1);
          for (int j = 0; j < boxes; ++j)
            tma_load_2d(dst + 2 * kHalfBytes + j * SH::BOX * 128, xm, bar, s * kSlab, w.row0 + j * SH::BOX);
        }
        __syncwarp();
      }
    }
    // the last products' arrivals find the CTA still there
    for (int s = max(0, n - STAGES); ok && s < n; ++s) ok = mbar_wait_or_fail(bar_empty + 8 * (s % STAGES), (s / STAGES) & 1);
    if (!ok) {
      if (lane == 0) *sfail = 1;
      // the copies in flight land before the CTA's memory goes away
      for (int s = max(0, n - STAGES); s < n; ++s) mbar_wait_or_fail(bar_full + 8 * (s % STAGES), (s / STAGES) & 1);
    }
  } else if (warp == 1) {
    // ===== MMA issuer =====
    const uint32_t tb = __shfl_sync(0xffffffffu, tmem, 0);
    int n = 0, it = 0;
    bool ok = true;
    for (int i = blockIdx.x; ok && i < work.total; i += gridDim.x, ++it) {
      const Item w = work.at(p, tiles, first, i);
      const int slabs = (w.k + kSlab - 1) / kSlab, b = it & 1;
      const bool both = GATED || w.feature + 128 < w.n_out;
      const uint32_t idesc = make_idesc(1, 128, (w.nrows + 15) & ~15);
      if (!(ok = mbar_wait_or_fail(bar_free + 8 * b, ((it >> 1) & 1) ^ 1))) break;
      const uint32_t d0 = tb + b * 2 * TOKENS, d1 = d0 + TOKENS;
      for (int s = 0; s < slabs; ++s, ++n) {
        const int st = n % STAGES;
        if (!(ok = mbar_wait_or_fail(bar_full + 8 * st, (n / STAGES) & 1))) break;
        tc_fence_after();
        if (elect_one()) {
          const uint32_t src = base + st * SH::STAGE_BYTES;
          const uint64_t a0 = make_smem_desc(src), a1 = make_smem_desc(src + kHalfBytes), x = make_smem_desc(src + 2 * kHalfBytes);
#pragma unroll
          for (int k = 0; k < kSlab / 16; ++k) {
            tc_mma_f16(d0, a0 + 2 * k, x + 2 * k, idesc, (s | k) != 0 ? 1u : 0u);
            if (both) tc_mma_f16(d1, a1 + 2 * k, x + 2 * k, idesc, (s | k) != 0 ? 1u : 0u);
          }
          tc_commit(bar_empty + 8 * st);
          if (s == slabs - 1) tc_commit(bar_acc + 8 * b);
        }
        __syncwarp();
      }
    }
    if (!ok && lane == 0) *sfail = 1;
  } else if (warp < 6) {
    // ===== epilogue =====
    const int q = warp & 3;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    int it = 0;
    bool ok = true;
    for (int i = blockIdx.x; i < work.total; i += gridDim.x, ++it) {
      const Item w = work.at(p, tiles, first, i);
      const int b = it & 1;
      if (!(ok = mbar_wait_or_fail(bar_acc + 8 * b, (it >> 1) & 1))) break;
      tc_fence_after();
      const uint32_t d0 = tmem + lane_addr + b * 2 * TOKENS, d1 = d0 + TOKENS;
      const int feature = w.feature + q * 32 + (lane & ~1);  // of the pair a lane stores
      __nv_bfloat16* out = (w.shared ? p.shared_out : p.out) + feature;
      const int64_t ost = w.shared ? p.shared_out_stride : p.out_stride;
      const bool live0 = feature < w.n_out, live1 = !GATED && feature + 128 < w.n_out, both = GATED || w.feature + 128 < w.n_out;
      for (int c0 = 0; c0 < w.nrows; c0 += 16) {
        uint32_t u[16], v[16];
        tmem_ld<16>(d0 + c0, u);
        if (both) tmem_ld<16>(d1 + c0, v);
        const int mine = w.row0 + min(c0 + (lane & 15), w.nrows - 1);
        const int place = GATED || w.shared ? mine : pair_at(mine);
        if (GATED) {
#pragma unroll
          for (int c = 0; c < 16; ++c) {
            const float z = __uint_as_float(u[c]);
            u[c] = __float_as_uint(z * __fdividef(1.f, 1.f + __expf(-z)) * __uint_as_float(v[c]));
          }
        }
        // neighbouring lanes swap a column each: one 4-byte store of two features a lane for two columns
#pragma unroll
        for (int c = 0; c < 16; c += 2) {
          const int col = c + (lane & 1), row = __shfl_sync(0xffffffffu, place, col);
          const bool live = c0 + col < w.nrows;
          __nv_bfloat16* o = out + row * ost;
          const uint32_t x = swap_pack(u[c], u[c + 1]);
          if (live && live0) *reinterpret_cast<uint32_t*>(o) = x;
          if (!GATED && both) {
            const uint32_t y = swap_pack(v[c], v[c + 1]);
            if (live && live1) *reinterpret_cast<uint32_t*>(o + 128) = y;
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_free + 8 * b);
    }
    if (!ok && lane == 0) *sfail = 1;
  } else if (GATED) {
    // ===== gathered token rows =====
    const int t = threadIdx.x - 192, c = t & 7, r_first = t >> 3;
    constexpr int PER = TOKENS / 16;
    int n = 0, arrived = 0;
    bool ok = true;
    auto arrive = [&] {
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_full + 8 * (arrived % STAGES));
      ++arrived;
    };
    for (int i = blockIdx.x; ok && i < work.total; i += gridDim.x) {
      const Item w = work.at(p, tiles, first, i);
      const int slabs = (w.k + kSlab - 1) / kSlab;
      const __nv_bfloat16* src[PER];
#pragma unroll
      for (int m = 0; m < PER; ++m) {
        const int r = r_first + 16 * m, row = w.row0 + min(r, w.nrows - 1);
        src[m] = p.x + (int64_t)(w.shared ? row : pair_at(row) / p.top) * p.x_stride + c * 8;
      }
      for (int s = 0; s < slabs; ++s) {
        const int st = n % STAGES;
        if (!(ok = mbar_wait_or_fail(bar_empty + 8 * st, ((n / STAGES) & 1) ^ 1))) break;
        const uint32_t dst = base + st * SH::STAGE_BYTES + 2 * kHalfBytes;
        const int bytes = s * kSlab + c * 8 < w.k ? 16 : 0;  // zeros past K
#pragma unroll
        for (int m = 0; m < PER; ++m) {
          const int r = r_first + 16 * m;
          if (r < w.nrows)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + r * 128 + ((c ^ (r & 7)) << 4)),
                         "l"(src[m] + (bytes ? s * kSlab : 0)), "r"(bytes) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        ++n;
        if (n - arrived == kGatherLag) {
          asm volatile("cp.async.wait_group %0;" ::"n"(kGatherLag - 1) : "memory");
          arrive();
        }
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    while (arrived < n) arrive();
    if (!ok && lane == 0) *sfail = 1;
  }
  tc_fence_before();
  __syncthreads();
  if (*sfail && threadIdx.x == 0) atomicExch(&g_failed, 1);
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(SH::TMEM_COLS) : "memory");
  }
}

inline bool supported(const b200_expert_product_args& a) {
  auto ok = [](const void* p, int64_t stride) { return !p || (((uintptr_t)p & 15) == 0 && stride % 8 == 0 && stride < (1ll << 36)); };
  return a.dtype == B200_BF16 && (a.tile_rows == 32 || a.tile_rows == 64 || a.tile_rows == 128) && a.k % 8 == 0 &&
         ok(a.x, a.x_stride) && ok(a.w, a.w_stride) && ok(a.out, a.out_stride) && ok(a.shared_out, a.shared_out_stride) &&
         (!a.shared_w || (a.shared_k % 8 == 0 && ok(a.shared_w, a.shared_w_stride) && ok(a.shared_x, a.shared_x_stride))) &&
         (int64_t)a.experts * a.n_out * 2 < (1ll << 31) && encode_fn() != nullptr;
}

template <int TOKENS, bool GATED>
int launch_form(const b200_expert_product_args& a, cudaStream_t st) {
  using SH = Shape<TOKENS>;
  auto kern = expert_product_tc_kernel<TOKENS, GATED>;
  const int smem = smem_bytes(SH::STAGES, SH::STAGE_BYTES, a.experts);
  static int configured[16] = {0};
  int dev = 0;
  B200_CUDA_OK(cudaGetDevice(&dev));
  if (configured[dev & 15] < smem) {
    B200_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    configured[dev & 15] = smem;
  }
  const CUtensorMapDataType bf = CU_TENSOR_MAP_DATA_TYPE_BFLOAT16;
  const CUtensorMapL2promotion promo = CU_TENSOR_MAP_L2_PROMOTION_L2_256B;
  CUtensorMap w, x, sw, sx;
  const int64_t w_rows = (int64_t)a.experts * a.n_out * (GATED ? 2 : 1);
  int rc = make_map_2d(&w, bf, a.w, a.k, w_rows, a.w_stride * 2, kSlab, 128, promo);
  if (rc == B200_OK && !GATED) rc = make_map_2d(&x, bf, a.x, a.k, (uint64_t)a.rows * a.top, a.x_stride * 2, kSlab, SH::BOX, promo);
  if (rc == B200_OK && a.shared_w) rc = make_map_2d(&sw, bf, a.shared_w, a.shared_k, (uint64_t)a.shared_n_out * (GATED ? 2 : 1),
                                                    a.shared_w_stride * 2, kSlab, 128, promo);
  if (rc == B200_OK && a.shared_w && !GATED)
    rc = make_map_2d(&sx, bf, a.shared_x, a.shared_k, a.rows, a.shared_x_stride * 2, kSlab, SH::BOX, promo);
  if (rc != B200_OK) return rc;
  if (GATED) x = sx = w;  // not read
  if (!a.shared_w) sw = w, sx = x;
  Params p;
  p.pairs = a.pairs;
  p.first = a.first;
  p.tiles = a.tiles;
  p.x = (const __nv_bfloat16*)a.x;
  p.out = (__nv_bfloat16*)a.out;
  p.shared_out = (__nv_bfloat16*)a.shared_out;
  p.x_stride = a.x_stride;
  p.out_stride = a.out_stride;
  p.shared_out_stride = a.shared_out_stride;
  p.rows = a.rows;
  p.experts = a.experts;
  p.top = a.top;
  p.n_out = a.n_out;
  p.k = a.k;
  p.shared_n_out = a.shared_n_out;
  p.shared_k = a.shared_k;
  p.max_tiles = a.max_tiles;
  p.shared_tiles = a.shared_w ? (a.rows + TOKENS - 1) / TOKENS : 0;
  constexpr int FEATURES = GATED ? 128 : 256;
  const int64_t items = (int64_t)a.max_tiles * ((a.n_out + FEATURES - 1) / FEATURES) +
                        (int64_t)p.shared_tiles * ((a.shared_n_out + FEATURES - 1) / FEATURES);
  const int sms = sm_count() > 0 ? sm_count() : 148;
  const int grid = items < sms ? (int)(items > 0 ? items : 1) : sms;
  B200_CUDA_OK(launch_pdl(kern, dim3(grid), dim3(GATED ? 320 : 192), smem, st, w, x, sw, sx, p));
  return check_launch("expert_product_tc_kernel");
}

inline int launch(const b200_expert_product_args& a, cudaStream_t st) {
  auto pick = [&](auto gated) {
    constexpr bool G = decltype(gated)::value;
    return a.tile_rows == 32 ? launch_form<32, G>(a, st) : a.tile_rows == 64 ? launch_form<64, G>(a, st) : launch_form<128, G>(a, st);
  };
  return a.gated ? pick(std::true_type()) : pick(std::false_type());
}

}  // namespace experts_tc
}  // namespace b200
