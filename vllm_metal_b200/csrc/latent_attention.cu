// Latent attention in the latent space over a paged cache (include/b200_hybrid_ops.h): all query heads of a token read
// the same cached row [latent | rotated key part], and the latent is the value as well, so a row is fetched once and
// used by heads x (scores + values).
//
//  * latent_mma_kernel (bf16): 32 (token, head) rows per CTA against 32-key tiles on m16n8k16 tensor cores, split over
//    the keys when the batch alone does not fill the GPU; softmax in fp32, the weights enter the value product as a
//    two-term bf16 split (16 significant bits).
//  * latent_tc_kernel (latent_attention_tc.cuh): the same on tcgen05, the default wherever pages and sizes allow TMA.
//  * latent_simt_kernel: any type and size; one CTA per (token, head).
#include "../../include/b200_hybrid_ops.h"
#include "latent_attention_tc.cuh"
#include "mma_sync.cuh"

namespace b200 {
namespace {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ int64_t slot_of(const b200_latent_attn_args& a, int s, int j) {
  return (int64_t)a.block_tables[(int64_t)s * a.max_blocks_per_seq + j / a.block_size] * a.block_size + j % a.block_size;
}

// ---- any type, any size -----------------------------------------------------------------------------
constexpr int kSimtThreads = 128;
constexpr int kSimtKeys = 64;
constexpr int kSimtRegs = 16;  // latent columns per thread: kv_rank <= 2048

template <typename T>
__global__ void __launch_bounds__(kSimtThreads)
latent_simt_kernel(const b200_latent_attn_args a) {
  extern __shared__ float sm[];
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.z, h = blockIdx.y, i = blockIdx.x;
  const int row0 = a.cu_seqlens[s], len = a.cu_seqlens[s + 1] - row0;
  if (i >= len || len > a.max_q_len) return;
  const int width = a.kv_rank + a.rot_dim, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  float* sq = sm;                // [width]
  float* sp = sq + width;        // [64]
  int* srow = reinterpret_cast<int*>(sp + kSimtKeys);
  const int pos = a.seq_lens[s] - len + i;
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0, hi = pos + 1;
  const T* q = reinterpret_cast<const T*>(a.q) + (int64_t)(row0 + i) * a.q_stride + (int64_t)h * width;
  const T* cache = reinterpret_cast<const T*>(a.cache);
  for (int d = tid; d < width; d += kSimtThreads) sq[d] = to_float(q[d]);
  float o[kSimtRegs];
#pragma unroll
  for (int r = 0; r < kSimtRegs; ++r) o[r] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int j0 = lo; j0 < hi; j0 += kSimtKeys) {
    const int n = min(kSimtKeys, hi - j0);
    __syncthreads();
    for (int j = tid; j < n; j += kSimtThreads) {
      const int64_t slot = slot_of(a, s, j0 + j);
      srow[j] = slot >= 0 && slot < a.num_slots ? (int)slot : 0;
    }
    __syncthreads();
    for (int j = warp; j < n; j += kSimtThreads / 32) {
      const T* c = cache + (int64_t)srow[j] * width;
      float acc = 0.f;
      for (int d = lane; d < width; d += 32) acc += sq[d] * to_float(c[d]);
      acc = warp_sum(acc);
      if (lane == 0) sp[j] = acc * a.scale;
    }
    __syncthreads();
    float mx = m;
    for (int j = 0; j < n; ++j) mx = fmaxf(mx, sp[j]);
    const float alpha = m == -INFINITY ? 0.f : expf(m - mx);
    m = mx;
    l *= alpha;
#pragma unroll
    for (int r = 0; r < kSimtRegs; ++r) o[r] *= alpha;
    for (int j = 0; j < n; ++j) {
      const float p = expf(sp[j] - m);
      l += p;
      const T* c = cache + (int64_t)srow[j] * width;
#pragma unroll
      for (int r = 0; r < kSimtRegs; ++r) {
        const int d = tid + r * kSimtThreads;
        if (d < a.kv_rank) o[r] += p * to_float(c[d]);
      }
    }
  }
  T* out = reinterpret_cast<T*>(a.out) + (int64_t)(row0 + i) * a.out_stride + (int64_t)h * a.kv_rank;
#pragma unroll
  for (int r = 0; r < kSimtRegs; ++r) {
    const int d = tid + r * kSimtThreads;
    if (d < a.kv_rank) out[d] = from_float<T>(o[r] / l);
  }
}

// ---- bf16 on tensor cores ----------------------------------------------------------------------
constexpr int kThreads = 256;
constexpr int kRows = 32, kKeys = 32;
constexpr int kPPitch = 40;
constexpr int kMaxRank = 512, kMaxWidth = 640, kMaxSplits = 64;

struct Smem {
  int pitch;
  size_t q, c, p, s, st, total;
  __host__ __device__ explicit Smem(int width) {
    pitch = width + 8;
    q = 0;
    c = q + (size_t)kRows * pitch * 2;
    p = c + 2 * (size_t)kKeys * pitch * 2;
    s = p + 2 * (size_t)kRows * kPPitch * 2;
    st = s + (size_t)kRows * 33 * 4;
    total = st + kRows * 4;
  }
};

__global__ void __launch_bounds__(kThreads, 2)
latent_mma_kernel(const b200_latent_attn_args a, int splits) {
  extern __shared__ __align__(16) uint8_t raw[];
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.y, split = blockIdx.z;
  const int row0 = a.cu_seqlens[s], len = a.cu_seqlens[s + 1] - row0;
  const int r_first = blockIdx.x * kRows;
  if (len <= 0 || len > a.max_q_len || r_first >= len * a.heads) return;
  const int rank = a.kv_rank, width = rank + a.rot_dim;
  const Smem lay(width);
  bf16* sq = reinterpret_cast<bf16*>(raw + lay.q);
  bf16* sc = reinterpret_cast<bf16*>(raw + lay.c);
  bf16* sp = reinterpret_cast<bf16*>(raw + lay.p);
  float* ss = reinterpret_cast<float*>(raw + lay.s);
  float* salpha = reinterpret_cast<float*>(raw + lay.st);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, pitch = lay.pitch;
  const int nrows = min(kRows, len * a.heads - r_first);
  const int start = a.seq_lens[s] - len;
  const int pos_first = start + r_first / a.heads, pos_last = start + (r_first + nrows - 1) / a.heads;
  const int lo_all = a.window > 0 ? max(0, pos_first - a.window + 1) : 0, hi_all = pos_last + 1;
  const int tiles = (hi_all - lo_all + kKeys - 1) / kKeys;
  const int t_begin = (int)((int64_t)tiles * split / splits), t_end = (int)((int64_t)tiles * (split + 1) / splits);
  const int chunks = width >> 3;
  const bf16* cache = reinterpret_cast<const bf16*>(a.cache);
  for (int i = tid; i < kRows * chunks; i += kThreads) {
    const int r = i / chunks, c = (i - r * chunks) * 8, rr = r_first + r;
    const bool live = r < nrows;
    const bf16* src = reinterpret_cast<const bf16*>(a.q);
    if (live) src += (int64_t)(row0 + rr / a.heads) * a.q_stride + (int64_t)(rr % a.heads) * width + c;
    mma::cp_async16(&sq[r * pitch + c], src, live);
  }
  auto fetch = [&](int t, int buf) {
    // 8 threads a key; a key's page is looked up once per thread
    const int j = tid >> 3, key = lo_all + t * kKeys + j;
    bool live = key < hi_all;
    const int64_t slot = live ? slot_of(a, s, key) : 0;
    live = live && slot >= 0 && slot < a.num_slots;
    const bf16* src = cache + (live ? slot : 0) * width;
    bf16* dst = sc + ((size_t)buf * kKeys + j) * pitch;
    for (int c = tid & 7; c < chunks; c += 8) mma::cp_async16(dst + c * 8, src + c * 8, live);
  };
  float o[4][2][2][4];  // [n16 of this warp][m16][n8][4]
#pragma unroll
  for (int x = 0; x < 4; ++x)
#pragma unroll
    for (int y = 0; y < 2; ++y)
#pragma unroll
      for (int z = 0; z < 2; ++z)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[x][y][z][e] = 0.f;
  float m_row[4], l_row[4];  // rows 4 * warp + i of the tile, every lane the same
#pragma unroll
  for (int i = 0; i < 4; ++i) m_row[i] = -INFINITY, l_row[i] = 0.f;
  if (t_begin < t_end) fetch(t_begin, 0);
  mma::cp_commit();
  const float scale2 = a.scale * kLog2e;
  const int ksteps = width >> 4;
  for (int t = t_begin; t < t_end; ++t) {
    const int buf = (t - t_begin) & 1;
    if (t + 1 < t_end) fetch(t + 1, buf ^ 1);
    mma::cp_commit();
    mma::cp_wait<1>();
    __syncthreads();
    const bf16* ct = sc + (size_t)buf * kKeys * pitch;
    {  // scores: warp -> m16 tile warp & 1, n8 tile warp >> 1
      float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
      const bf16* qa = sq + ((warp & 1) * 16 + (lane & 15)) * pitch + (lane >> 4) * 8;
      const bf16* kb = ct + ((warp >> 1) * 8 + (lane & 7)) * pitch + (lane >> 3) * 8;
      int ks = 0;
      for (; ks + 1 < ksteps; ks += 2) {
        uint32_t fa[4], fa2[4], fb[4];
        mma::ldsm4(fa, qa + ks * 16);
        mma::ldsm4(fa2, qa + ks * 16 + 16);
        mma::ldsm4(fb, kb + ks * 16);
        mma::mma16816(acc[0], fa, fb[0], fb[1]);
        mma::mma16816(acc[1], fa2, fb[2], fb[3]);
      }
      if (ks < ksteps) {
        uint32_t fa[4], fb[4];
        mma::ldsm4(fa, qa + ks * 16);
        mma::ldsm4(fb, ct + ((warp >> 1) * 8 + (lane & 7)) * pitch + ((lane >> 3) & 1) * 8 + ks * 16);
        mma::mma16816(acc[0], fa, fb[0], fb[1]);
      }
      const int r = (warp & 1) * 16 + (lane >> 2), c = (warp >> 1) * 8 + (lane & 3) * 2;
      ss[r * 33 + c] = acc[0][0] + acc[1][0];
      ss[r * 33 + c + 1] = acc[0][1] + acc[1][1];
      ss[(r + 8) * 33 + c] = acc[0][2] + acc[1][2];
      ss[(r + 8) * 33 + c + 1] = acc[0][3] + acc[1][3];
    }
    __syncthreads();
    {  // softmax: 4 rows a warp, one key a lane
      const int key = lo_all + t * kKeys + lane;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = warp * 4 + i, pos = start + (r_first + r) / a.heads;
        const bool see = r < nrows && key <= pos && (a.window <= 0 || pos - key < a.window);
        const float x = see ? ss[r * 33 + lane] * scale2 : -INFINITY;
        const float mx = fmaxf(m_row[i], warp_max(x));
        const float p = mx == -INFINITY ? 0.f : exp2f(x - mx);
        const float alpha = mx == -INFINITY ? 1.f : exp2f(m_row[i] - mx);
        l_row[i] = l_row[i] * alpha + warp_sum(p);
        m_row[i] = mx;
        const bf16 p_hi = __float2bfloat16_rn(p);
        sp[r * kPPitch + lane] = p_hi;
        sp[(kRows + r) * kPPitch + lane] = __float2bfloat16_rn(p - __bfloat162float(p_hi));
        if (lane == 0) salpha[r] = alpha;
      }
    }
    __syncthreads();
    uint32_t fp[2][2][2][4];  // [term][m16][k16]
#pragma unroll
    for (int term = 0; term < 2; ++term)
#pragma unroll
      for (int mt = 0; mt < 2; ++mt)
#pragma unroll
        for (int ks = 0; ks < 2; ++ks)
          mma::ldsm4(fp[term][mt][ks], sp + (term * kRows + mt * 16 + (lane & 15)) * kPPitch + ks * 16 + (lane >> 4) * 8);
    float al[2][2];
#pragma unroll
    for (int mt = 0; mt < 2; ++mt) {
      al[mt][0] = salpha[mt * 16 + (lane >> 2)];
      al[mt][1] = salpha[mt * 16 + (lane >> 2) + 8];
    }
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int col = (x * 8 + warp) * 16;
      if (col >= rank) break;
#pragma unroll
      for (int mt = 0; mt < 2; ++mt)
#pragma unroll
        for (int z = 0; z < 2; ++z)
#pragma unroll
          for (int e = 0; e < 4; ++e) o[x][mt][z][e] *= al[mt][e >> 1];
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        uint32_t fb[4];
        mma::ldsm4t(fb, ct + (ks * 16 + (lane & 15)) * pitch + col + (lane >> 4) * 8);
#pragma unroll
        for (int mt = 0; mt < 2; ++mt)
#pragma unroll
          for (int term = 0; term < 2; ++term) {
            mma::mma16816(o[x][mt][0], fp[term][mt][ks], fb[0], fb[1]);
            mma::mma16816(o[x][mt][1], fp[term][mt][ks], fb[2], fb[3]);
          }
      }
    }
    __syncthreads();
  }
  mma::cp_wait<0>();
  // rows' l (single pass) or nothing (split): the divisor goes through salpha
#pragma unroll
  for (int i = 0; i < 4; ++i)
    if (lane == 0) salpha[warp * 4 + i] = splits == 1 ? 1.f / l_row[i] : 1.f;
  float* wo = reinterpret_cast<float*>(a.workspace);
  const size_t all_rows = (size_t)a.num_tokens * a.heads;
  float* wml = wo + (size_t)splits * all_rows * rank;
  const size_t base = (size_t)row0 * a.heads + r_first;
  if (splits > 1 && lane == 0)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = warp * 4 + i;
      if (r < nrows) {
        wml[2 * (split * all_rows + base + r)] = m_row[i];
        wml[2 * (split * all_rows + base + r) + 1] = l_row[i];
      }
    }
  __syncthreads();
#pragma unroll
  for (int x = 0; x < 4; ++x) {
    if ((x * 8 + warp) * 16 >= rank) break;
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
      for (int z = 0; z < 2; ++z)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = mt * 16 + (lane >> 2) + e * 8, col = (x * 8 + warp) * 16 + z * 8 + (lane & 3) * 2;
          if (r >= nrows) continue;
          const float inv = salpha[r], u = o[x][mt][z][2 * e] * inv, v = o[x][mt][z][2 * e + 1] * inv;
          const int rr = r_first + r;
          if (splits == 1)
            *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<bf16*>(a.out) + (int64_t)(row0 + rr / a.heads) * a.out_stride +
                                               (int64_t)(rr % a.heads) * rank + col) = __floats2bfloat162_rn(u, v);
          else
            *reinterpret_cast<float2*>(wo + (split * all_rows + base + r) * rank + col) = make_float2(u, v);
        }
  }
}

// The splits' partial outputs of a (token, head) row become one: `wpr` warps a row, 4 columns a lane and step.
__global__ void __launch_bounds__(256)
latent_merge_kernel(const b200_latent_attn_args a, int splits, int wpr) {
  pdl_trigger();
  pdl_wait();
  __shared__ float weights[8][kMaxSplits];
  const int s = blockIdx.y, row0 = a.cu_seqlens[s], len = a.cu_seqlens[s + 1] - row0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rr = blockIdx.x * (8 / wpr) + warp / wpr;
  if (len <= 0 || len > a.max_q_len || rr >= len * a.heads) return;
  const int rank = a.kv_rank;
  const size_t all_rows = (size_t)a.num_tokens * a.heads, row = (size_t)row0 * a.heads + rr;
  const float* wo = reinterpret_cast<const float*>(a.workspace);
  const float2* wml = reinterpret_cast<const float2*>(wo + (size_t)splits * all_rows * rank);
  float* weight = weights[warp];
  float m = -INFINITY, l = 0.f;
  for (int p = lane; p < splits; p += 32) m = fmaxf(m, wml[p * all_rows + row].x);
  m = warp_max(m);
  for (int p = lane; p < splits; p += 32) {
    const float2 ml = wml[p * all_rows + row];
    const float w = ml.x == -INFINITY ? 0.f : exp2f(ml.x - m);
    weight[p] = w;
    l += w * ml.y;
  }
  l = warp_sum(l);
  __syncwarp();
  const float inv = 1.f / l;
  bf16* out = reinterpret_cast<bf16*>(a.out) + (int64_t)(row0 + rr / a.heads) * a.out_stride + (int64_t)(rr % a.heads) * rank;
#pragma unroll 4
  for (int d = (warp % wpr) * 128 + lane * 4; d < rank; d += wpr * 128) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 2
    for (int p = 0; p < splits; ++p) {
      const float w = weight[p];
      const float4 v = *reinterpret_cast<const float4*>(wo + (p * all_rows + row) * rank + d);
      acc.x += w * v.x, acc.y += w * v.y, acc.z += w * v.z, acc.w += w * v.w;
    }
    reinterpret_cast<__nv_bfloat162*>(out + d)[0] = __floats2bfloat162_rn(acc.x * inv, acc.y * inv);
    reinterpret_cast<__nv_bfloat162*>(out + d)[1] = __floats2bfloat162_rn(acc.z * inv, acc.w * inv);
  }
}

enum Kind { kSimt = 1, kMma = 2, kTc = 3 };
struct Plan {
  Kind kind;
  int splits;
};

bool tc_supported(const b200_latent_attn_args& a) {
  const int width = a.kv_rank + a.rot_dim;
  return a.dtype == B200_BF16 && a.scale > 0.f && width % 8 == 0 && a.kv_rank % 8 == 0 && a.kv_rank <= kMaxRank &&
         width <= 64 * latent_tc::kMaxSlices && a.q_stride == (int64_t)a.heads * width &&
         a.out_stride == (int64_t)a.heads * a.kv_rank && a.block_size >= 8 &&
         latent_tc::kKeys % a.block_size == 0 && a.num_slots < (1LL << 31) &&
         (((uintptr_t)a.q | (uintptr_t)a.cache) & 15) == 0 && tc::encode_fn() != nullptr;
}

bool mma_supported(const b200_latent_attn_args& a) {
  const int width = a.kv_rank + a.rot_dim;
  return a.dtype == B200_BF16 && a.kv_rank % 16 == 0 && width % 16 == 0 && a.kv_rank <= kMaxRank && width <= kMaxWidth &&
         a.q_stride % 8 == 0 && a.out_stride % 8 == 0 &&
         (((uintptr_t)a.q | (uintptr_t)a.cache | (uintptr_t)a.out) & 15) == 0;
}

Plan plan(const b200_latent_attn_args& a) {
  Plan p{kSimt, 1};
  if ((a.kernel == 0 || a.kernel == kTc) && tc_supported(a))
    p.kind = kTc;
  else if ((a.kernel == 0 || a.kernel == kMma) && mma_supported(a))
    p.kind = kMma;
  if (p.kind == kSimt) return p;
  const int64_t items = (int64_t)a.num_seqs * ((a.max_q_len * a.heads + kRows - 1) / kRows);
  int keys = a.max_seq_len;
  if (a.window > 0 && a.window + a.max_q_len < keys) keys = a.window + a.max_q_len;
  const int tile = p.kind == kTc ? latent_tc::kKeys : kKeys;
  const int tiles = (keys + tile - 1) / tile;
  if (a.force_splits > 0) {
    p.splits = a.force_splits < tiles ? a.force_splits : (tiles > 0 ? tiles : 1);
    if (p.splits > kMaxSplits) p.splits = kMaxSplits;
    return p;
  }
  // waves of resident CTAs; a wave costs its tiles plus a fill / drain of about 3, a split adds the merge launch
  const int64_t resident = (p.kind == kTc ? 1 : 2) * (int64_t)(sm_count() > 0 ? sm_count() : 148);
  double best = 1e30;
  for (int s = 1; s <= kMaxSplits && s * 2 <= (tiles > 2 ? tiles : 2); ++s) {
    const double waves = (double)((items * s + resident - 1) / resident);
    const double cost = waves * ((tiles + s - 1) / s + 3.0) + (s > 1 ? 3.0 + 0.1 * s : 0.0);
    if (cost < best) best = cost, p.splits = s;
  }
  return p;
}

int launch_tc(const b200_latent_attn_args& a, int splits, cudaStream_t st) {
  using namespace latent_tc;
  Params p;
  p.block_tables = a.block_tables, p.seq_lens = a.seq_lens, p.cu = a.cu_seqlens, p.out = a.out;
  p.wo = reinterpret_cast<float*>(a.workspace);
  p.num_tokens = a.num_tokens, p.heads = a.heads, p.rank = a.kv_rank;
  p.width = a.kv_rank + a.rot_dim, p.slices = (p.width + 63) / 64, p.mtiles = (a.kv_rank + 127) / 128;
  p.block_size = a.block_size, p.max_blocks = a.max_blocks_per_seq, p.window = a.window, p.max_q_len = a.max_q_len;
  p.splits = splits, p.scale2 = a.scale * kLog2e;
  CUtensorMap q_map, c_map;
  int rc = tc::make_map_2d(&q_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, a.q, p.width, (uint64_t)a.num_tokens * a.heads,
                           (uint64_t)p.width * 2, 64, latent_tc::kRows, CU_TENSOR_MAP_L2_PROMOTION_L2_128B);
  if (rc != B200_OK) return rc;
  rc = tc::make_map_2d(&c_map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, a.cache, p.width, (uint64_t)a.num_slots,
                       (uint64_t)p.width * 2, 64, a.block_size, CU_TENSOR_MAP_L2_PROMOTION_L2_128B);
  if (rc != B200_OK) return rc;
  static bool attr = false;
  if (!attr) {
    B200_CUDA_OK(cudaFuncSetAttribute(latent_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                      latent_tc::smem_bytes(latent_tc::kMaxSlices)));
    attr = true;
  }
  const int rows = a.max_q_len * a.heads;
  B200_CUDA_OK(launch_pdl(latent_tc_kernel, dim3((rows + latent_tc::kRows - 1) / latent_tc::kRows, a.num_seqs, splits),
                          dim3(latent_tc::kThreads), latent_tc::smem_bytes(p.slices), st, q_map, c_map, p));
  return B200_OK;
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

size_t b200_latent_attention_workspace_bytes(const b200_latent_attn_args* a) {
  if (!a) return 0;
  const Plan p = plan(*a);
  return p.splits > 1 ? (size_t)p.splits * a->num_tokens * a->heads * (a->kv_rank + 2) * sizeof(float) : 0;
}

int b200_latent_attention_num_launches(const b200_latent_attn_args* a) {
  return plan(*a).splits > 1 ? 2 : 1;
}

int b200_latent_attention(const b200_latent_attn_args* a, void* stream) {
  B200_CHECK_ARG(a && a->q && a->cache && a->block_tables && a->seq_lens && a->cu_seqlens && a->out,
                 "latent_attention: null argument");
  B200_CHECK_ARG(a->heads > 0 && a->kv_rank > 0 && a->rot_dim >= 0 && a->block_size > 0 && a->num_slots > 0,
                 "latent_attention: bad sizes");
  if (a->num_tokens <= 0 || a->num_seqs <= 0 || a->max_q_len <= 0) return B200_OK;
  B200_CHECK_ARG(a->num_seqs <= 65535, "latent_attention: batch too large");
  cudaStream_t st = (cudaStream_t)stream;
  const Plan p = plan(*a);
  if (p.kind == kSimt) {
    B200_CHECK_ARG(a->kernel <= 1, "latent_attention: this type or these sizes have no tensor-core form");
    B200_CHECK_ARG(a->kv_rank <= kSimtThreads * kSimtRegs, "latent_attention: kv_rank %d above %d", a->kv_rank,
                   kSimtThreads * kSimtRegs);
    B200_CHECK_ARG(a->heads <= 65535 && a->num_slots < (1LL << 31), "latent_attention: batch too large");
    const size_t smem = (size_t)(a->kv_rank + a->rot_dim + 2 * kSimtKeys) * 4;
    return B200_DISPATCH_DTYPE(a->dtype, T, [&]() -> int {
      B200_CUDA_OK(launch_pdl(latent_simt_kernel<T>, dim3(a->max_q_len, a->heads, a->num_seqs), dim3(kSimtThreads),
                              smem, st, *a));
      return check_launch("latent_attention (simt)");
    });
  }
  B200_CHECK_ARG(b200_latent_attention_workspace_bytes(a) <= a->workspace_bytes, "latent_attention: workspace too small");
  const int rows = a->max_q_len * a->heads;
  static bool attr = false;
  if (p.kind == kTc) {
    const int rc = launch_tc(*a, p.splits, st);
    if (rc != B200_OK) return rc;
  } else if (!attr) {
    B200_CUDA_OK(cudaFuncSetAttribute(latent_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                      (int)Smem(kMaxWidth).total));
    attr = true;
  }
  if (p.kind == kMma)
    B200_CUDA_OK(launch_pdl(latent_mma_kernel, dim3((rows + kRows - 1) / kRows, a->num_seqs, p.splits), dim3(kThreads),
                          Smem(a->kv_rank + a->rot_dim).total, st, *a, p.splits));
  if (p.splits > 1) {
    const int wpr = (int64_t)rows * a->num_seqs >= 1024 ? 1 : 4;
    B200_CUDA_OK(launch_pdl(latent_merge_kernel, dim3((rows * wpr + 7) / 8, a->num_seqs), dim3(256), 0, st, *a, p.splits, wpr));
  }
  return check_launch("latent_attention");
}

// 1 if a bounded wait of the tcgen05 kernel ever ran out in this process (its results were then not written).
int b200_latent_attention_failed(void) {
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, latent_tc::g_failed, sizeof(v)) != cudaSuccess) return -1;
  return v;
}

}  // extern "C"
