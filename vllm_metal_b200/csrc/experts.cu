// Routed experts (include/b200_hybrid_ops.h): routing, the sort of (row, place) pairs by expert, and the products of all
// experts at once -- on tcgen05 (experts_tc.cuh) or, for any type and size, the tile kernel here.  Nothing is read back to
// the host: grids are bounds, the work is found from the plan on the device.
#include "../../include/b200_hybrid_ops.h"
#include "experts_tc.cuh"
#include "row_ops.cuh"

namespace b200 {
namespace {

// No __restrict__ on what an earlier launch writes: it would make the loads read-only ones, which are not held back by
// the wait for that launch.

// ---- routing: a warp per row ------------------------------------------------------------------------
constexpr int kRouteWarps = 4;

__global__ void __launch_bounds__(kRouteWarps * 32)
expert_route_kernel(const float* logits, int64_t stride, const float* correction, int32_t* chosen, float* weights, int rows,
                    int experts, int top, float scale, int over_chosen) {
  extern __shared__ float sm[];  // per warp: scores [experts], choice scores [experts]
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t r = (int64_t)blockIdx.x * kRouteWarps + warp;
  if (r >= rows) return;
  float* s = sm + warp * 2 * experts;
  float* c = s + experts;
  float m = -INFINITY;
  for (int e = lane; e < experts; e += 32) {
    s[e] = logits[r * stride + e];
    if (over_chosen) c[e] = s[e] = s[e] + (correction ? correction[e] : 0.f);
    m = fmaxf(m, s[e]);
  }
  m = warp_max(m);
  float sum = 0.f;
  for (int e = lane; e < experts; e += 32) {
    s[e] = expf(s[e] - m);
    sum += s[e];
  }
  const float inv = over_chosen ? 1.f : 1.f / warp_sum(sum);
  float best = -INFINITY;  // this lane's best remaining one; it alone looks at its experts again
  int at = 0x7fffffff;
  auto look = [&] {
    best = -INFINITY;
    at = 0x7fffffff;
    for (int e = lane; e < experts; e += 32)
      if (c[e] > best) best = c[e], at = e;
  };
  for (int e = lane; e < experts; e += 32) {
    s[e] *= inv;
    if (!over_chosen) c[e] = s[e] + (correction ? correction[e] : 0.f);
  }
  look();
  float taken = 0.f;  // on the lane of each choice
  for (int j = 0; j < top; ++j) {
    const uint32_t bits = __float_as_uint(best), key = bits ^ ((int32_t)bits < 0 ? 0xffffffffu : 0x80000000u);  // same order
    const uint32_t top_key = __reduce_max_sync(0xffffffffu, key);
    int i = __reduce_min_sync(0xffffffffu, key == top_key ? at : 0x7fffffff);
    if (i >= experts) i = j % experts;  // scores that compare with nothing (NaN): any expert, in bounds
    if (lane == i % 32) {
      chosen[r * top + j] = i;
      weights[r * top + j] = s[i] * scale;
      taken += s[i];
      c[i] = -INFINITY;
      look();
    }
  }
  if (over_chosen) {
    const float f = 1.f / warp_sum(taken);
    __syncwarp();
    for (int j = lane; j < top; j += 32) weights[r * top + j] *= f;
  }
}

// ---- plan: pairs sorted by expert, one CTA ----------------------------------------------------------
constexpr int kPlanThreads = 1024, kPlanKeep = 16;

__global__ void __launch_bounds__(kPlanThreads)
expert_plan_kernel(const int32_t* chosen, int32_t* pairs, int32_t* first, int32_t* tiles, int total, int experts, int tile_rows) {
  extern __shared__ int count[];  // [experts] counts, then next free places
  __shared__ int warp_pairs[32], warp_tiles[32], base_pairs, base_tiles;
  pdl_trigger();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  for (int e = tid; e < experts; e += kPlanThreads) count[e] = 0;
  if (tid == 0) base_pairs = base_tiles = 0;
  pdl_wait();
  __syncthreads();
  auto expert_of = [&](int p) { return min((uint32_t)chosen[p], (uint32_t)experts - 1); };  // in bounds whatever it holds
  // up to kPlanKeep pairs a thread stay in registers for the second pass
  int keep[kPlanKeep];
#pragma unroll
  for (int j = 0; j < kPlanKeep; ++j) {
    const int p = tid + j * kPlanThreads;
    keep[j] = p < total ? (int)expert_of(p) : -1;
  }
#pragma unroll
  for (int j = 0; j < kPlanKeep; ++j)
    if (keep[j] >= 0) atomicAdd(&count[keep[j]], 1);
  for (int p = tid + kPlanKeep * kPlanThreads; p < total; p += kPlanThreads) atomicAdd(&count[expert_of(p)], 1);
  __syncthreads();
  for (int e0 = 0; e0 < experts; e0 += kPlanThreads) {  // running sums, kPlanThreads experts at a time
    const int e = e0 + tid, n = e < experts ? count[e] : 0, nt = (n + tile_rows - 1) / tile_rows;
    int sp = n, st = nt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int ap = __shfl_up_sync(0xffffffffu, sp, o), at = __shfl_up_sync(0xffffffffu, st, o);
      if (lane >= o) sp += ap, st += at;
    }
    if (lane == 31) warp_pairs[warp] = sp, warp_tiles[warp] = st;
    __syncthreads();
    int bp = base_pairs, bt = base_tiles;
    for (int w = 0; w < warp; ++w) bp += warp_pairs[w], bt += warp_tiles[w];
    if (e < experts) {
      first[e] = count[e] = bp + sp - n;
      tiles[e] = bt + st - nt;
    }
    __syncthreads();
    if (tid == kPlanThreads - 1) base_pairs = bp + sp, base_tiles = bt + st;
    __syncthreads();
  }
  if (tid == 0) first[experts] = base_pairs, tiles[experts] = base_tiles;
  // places inside a stretch are taken as they come: a pair's results do not depend on its place
#pragma unroll
  for (int j = 0; j < kPlanKeep; ++j)
    if (keep[j] >= 0) pairs[atomicAdd(&count[keep[j]], 1)] = tid + j * kPlanThreads;
  for (int p = tid + kPlanKeep * kPlanThreads; p < total; p += kPlanThreads) pairs[atomicAdd(&count[expert_of(p)], 1)] = p;
}

// ---- products, any type and size ----------------------------------------------------------------------
constexpr int kSimtRows = 32, kSimtCols = 32, kSimtK = 32;

template <typename T, bool GATED>
__global__ void __launch_bounds__(256)
expert_product_kernel(const b200_expert_product_args a) {
  __shared__ float xs[kSimtK][kSimtRows + 1], ws[GATED ? 2 : 1][kSimtK][kSimtCols + 1];
  __shared__ int64_t src[kSimtRows], dst[kSimtRows];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x;
  const bool shared = a.shared_w && blockIdx.z == 1;
  const int n_out = shared ? a.shared_n_out : a.n_out, k_dim = shared ? a.shared_k : a.k;
  const int col0 = blockIdx.x * kSimtCols;
  if (col0 >= n_out) return;
  int row0 = 0, nrows = 0;
  int64_t w_row = 0;
  if (shared) {
    row0 = blockIdx.y * kSimtRows;
    nrows = min(kSimtRows, a.rows - row0);
  } else {
    const int tile = blockIdx.y;
    if (tile >= a.tiles[a.experts]) return;
    const int e = find_stretch(a.tiles, a.experts, tile);
    row0 = a.first[e] + (tile - a.tiles[e]) * kSimtRows;
    nrows = min(kSimtRows, a.first[e + 1] - row0);
    w_row = (int64_t)e * n_out * (GATED ? 2 : 1);
  }
  if (nrows <= 0) return;
  if (tid < kSimtRows) {
    const int i = row0 + min(tid, nrows - 1);
    const int pair = shared ? i : a.pairs[i];
    src[tid] = (GATED ? (shared ? i : pair / a.top) : i);
    dst[tid] = GATED ? i : pair;
  }
  __syncthreads();
  const T* x = reinterpret_cast<const T*>(shared && !GATED ? a.shared_x : a.x);
  const int64_t xst = shared && !GATED ? a.shared_x_stride : a.x_stride;
  const T* w = reinterpret_cast<const T*>(shared ? a.shared_w : a.w);
  const int64_t wst = shared ? a.shared_w_stride : a.w_stride;
  const int r = tid / 8, c4 = (tid % 8) * 4;  // a row and four columns each
  float acc[GATED ? 2 : 1][4] = {};
  for (int k0 = 0; k0 < k_dim; k0 += kSimtK) {
    for (int i = tid; i < kSimtRows * kSimtK; i += 256) {
      const int rr = i / kSimtK, kk = i % kSimtK;
      xs[kk][rr] = k0 + kk < k_dim ? to_float(x[src[rr] * xst + k0 + kk]) : 0.f;
    }
#pragma unroll
    for (int g = 0; g < (GATED ? 2 : 1); ++g)
      for (int i = tid; i < kSimtCols * kSimtK; i += 256) {
        const int cc = i / kSimtK, kk = i % kSimtK;
        ws[g][kk][cc] = k0 + kk < k_dim && col0 + cc < n_out ? to_float(w[(w_row + (int64_t)g * n_out + col0 + cc) * wst + k0 + kk]) : 0.f;
      }
    __syncthreads();
#pragma unroll 8
    for (int kk = 0; kk < kSimtK; ++kk) {
      const float v = xs[kk][r];
#pragma unroll
      for (int g = 0; g < (GATED ? 2 : 1); ++g)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[g][j] = fmaf(v, ws[g][kk][c4 + j], acc[g][j]);
    }
    __syncthreads();
  }
  if (r >= nrows) return;
  T* out = reinterpret_cast<T*>(shared ? a.shared_out : a.out) + dst[r] * (shared ? a.shared_out_stride : a.out_stride);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int c = col0 + c4 + j;
    if (c >= n_out) continue;
    float v = acc[0][j];
    if (GATED) v = v * gate_f(v) * acc[GATED ? 1 : 0][j];
    out[c] = from_float<T>(v);
  }
}

template <typename T>
int launch_simt(const b200_expert_product_args& a, cudaStream_t st) {
  const int cols = a.shared_w && a.shared_n_out > a.n_out ? a.shared_n_out : a.n_out;
  const int shared_tiles = a.shared_w ? (a.rows + kSimtRows - 1) / kSimtRows : 0;
  const int ty = a.max_tiles > shared_tiles ? a.max_tiles : shared_tiles;
  B200_CHECK_ARG(ty <= 65535, "expert_product: too many rows");
  const dim3 grid((cols + kSimtCols - 1) / kSimtCols, ty, a.shared_w ? 2 : 1);
  B200_CUDA_OK(launch_pdl(a.gated ? expert_product_kernel<T, true> : expert_product_kernel<T, false>, grid, dim3(256), 0, st, a));
  return check_launch("expert_product");
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_expert_route(const float* logits, int64_t logits_stride, const float* correction, int32_t* chosen, float* weights,
                      int rows, int experts, int top, float scale, int over_chosen, void* stream) {
  B200_CHECK_ARG(logits && chosen && weights, "expert_route: null pointer argument");
  B200_CHECK_ARG(experts >= 1 && experts <= B200_MAX_EXPERTS && top >= 1 && top <= experts,
                 "expert_route: %d of %d experts (at most %d)", top, experts, B200_MAX_EXPERTS);
  if (rows <= 0) return B200_OK;
  B200_CUDA_OK(launch_pdl(expert_route_kernel, dim3((rows + kRouteWarps - 1) / kRouteWarps), dim3(kRouteWarps * 32),
                          (size_t)kRouteWarps * 2 * experts * sizeof(float), (cudaStream_t)stream, logits, logits_stride,
                          correction, chosen, weights, rows, experts, top, scale, over_chosen));
  return check_launch("expert_route");
}

int b200_expert_plan(const int32_t* chosen, int32_t* pairs, int32_t* first, int32_t* tiles, int rows, int experts, int top,
                     int tile_rows, void* stream) {
  B200_CHECK_ARG(chosen && pairs && first && tiles, "expert_plan: null pointer argument");
  B200_CHECK_ARG(experts >= 1 && experts <= B200_MAX_EXPERTS && top >= 1 && tile_rows >= 1, "expert_plan: bad sizes");
  B200_CHECK_ARG((int64_t)rows * top < (1ll << 31), "expert_plan: too many pairs");
  B200_CUDA_OK(launch_pdl(expert_plan_kernel, dim3(1), dim3(kPlanThreads), (size_t)experts * sizeof(int), (cudaStream_t)stream,
                          chosen, pairs, first, tiles, rows * top, experts, tile_rows));
  return check_launch("expert_plan");
}

int b200_expert_product(const b200_expert_product_args* a, void* stream) {
  B200_CHECK_ARG(a && a->x && a->w && a->out && a->pairs && a->first && a->tiles, "expert_product: null pointer argument");
  B200_CHECK_ARG(a->experts >= 1 && a->experts <= B200_MAX_EXPERTS && a->top >= 1 && a->n_out >= 1 && a->k >= 1 && a->max_tiles >= 0,
                 "expert_product: bad sizes");
  B200_CHECK_ARG(!a->shared_w || (a->shared_out && a->shared_n_out >= 1 && a->shared_k >= 1 && (a->gated || a->shared_x)),
                 "expert_product: a shared expert without its operands");
  if (a->rows <= 0) return B200_OK;
  const bool tc = a->kernel != 1 && experts_tc::supported(*a);
  if (a->kernel == 2 && !tc)
    return set_error(B200_ERR_UNSUPPORTED, "expert_product: the tcgen05 kernel needs bf16, whole 8-element units, 16-byte aligned "
                     "operands and tiles of 32, 64 or 128 rows");
  if (tc) return experts_tc::launch(*a, (cudaStream_t)stream);
  B200_CHECK_ARG(a->tile_rows == kSimtRows, "expert_product: the any-size kernel takes tiles of %d rows, got %d", kSimtRows, a->tile_rows);
  return B200_DISPATCH_DTYPE(a->dtype, T, [&]() -> int { return launch_simt<T>(*a, (cudaStream_t)stream); });
}

int b200_expert_product_failed(void) {
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, experts_tc::g_failed, sizeof(v)) != cudaSuccess) return 1;
  return v;
}

}  // extern "C"
