// Chunked form of the recurrence whose decay is a vector per row (kind 3), 64-row chunks in three launches as in
// recurrence_chunk.cuh; the scan is shared.
//
// Between a row s and a later row t a key channel decays by w_(s+1) .. w_(t-1).  A quotient of cumulative products would
// overflow where decays are strong, so a chunk is cut into blocks of 16 rows and only products of decays are ever formed:
//   up to a block's end      K_s = k_s * prod of the block's later decays
//   from a block's start     R_t = r_t * prod of the block's earlier decays
//   over a whole block       D_j
// A row of block i meets a row of an earlier block j through R_t D_(i-1) .. D_(j+1) K_s: tensor-core products, the D's
// multiplied into R on the way back through the blocks; after the first block R meets the state on entry.  Within a block the
// scores are formed in fp32 by the ordinary cores, a lane holding one k_s that decays as the rows go by.  The chunk's own
// contribution is built up block by block: U <- diag(D_j) U + K_j^T v_j.
//
// r, k, v are bf16; every 32-bit factor enters the products as a three-term split, products of two split factors as
// their six largest terms (24 significant bits).
#pragma once

#include "recurrence_chunk.cuh"

namespace b200 {
namespace rec {
namespace wkv {

constexpr int kThreads = 256;
constexpr int kBlock = 16, kBlocks = kChunk / kBlock;  // two warps a block
constexpr int kPitch = 68;                              // of fp32 tiles
constexpr int kFloatTile = kChunk * kPitch;

// As rec::load_tile, by all threads here.
__device__ __forceinline__ void load_rows(bf16* dst, const bf16* src, int64_t stride, int rows, int cols) {
#pragma unroll
  for (int i = threadIdx.x; i < 64 * 8; i += kThreads) {
    const int r = i >> 3, c = (i & 7) * 8;
    const bool live = r < rows && c < cols;
    mma::cp_async16(dst + r * kPad + c, live ? src + (int64_t)r * stride + c : src, live);
  }
}

struct Decays {  // of one key channel over a block
  float w[kBlock];
  __device__ __forceinline__ void load(const b200_recurrence_args& a, int row0, int rows, int first, int channel, bool live) {
    if (!live) {
#pragma unroll
      for (int i = 0; i < kBlock; ++i) w[i] = 1.f;
      return;
    }
    const float bias = a.bias_a[channel];
    const float* z = reinterpret_cast<const float*>(a.gate_a) + (int64_t)(row0 + first) * a.gate_stride + channel;
#pragma unroll
    for (int i = 0; i < kBlock; ++i) w[i] = first + i < rows ? z[i * a.gate_stride] : 0.f;
#pragma unroll
    for (int i = 0; i < kBlock; ++i) w[i] = first + i < rows ? expf(-expf(w[i] + bias)) : 1.f;  // rows past the end: no decay
  }
};

// K_s of one channel and block, split, into the term tiles; returns D.
__device__ __forceinline__ float keys_to_block_end(const Decays& d, const bf16* sk, bf16* split, int first, int n) {
  float run = 1.f;
#pragma unroll
  for (int i = kBlock - 1; i >= 0; --i) {
    const int at = (first + i) * kPad + n;
    float x = to_float(sk[at]) * run;
#pragma unroll
    for (int j = 0; j < kTerms; ++j) {
      const bf16 b = __float2bfloat16_rn(x);
      split[j * kTileElems + at] = b;
      x -= to_float(b);
    }
    run *= d.w[i];
  }
  return run;
}

// ---- 1: a chunk's own contribution and its decay -----------------------------------------------------
// A CTA has one slab of key channels; the value tiles pass by it.
constexpr int kStateSmem = (3 + kTerms) * kTileElems * 2 + kBlocks * 64 * 4;

__global__ void __launch_bounds__(kThreads, 3)
state_kernel(const b200_recurrence_args a) {
  extern __shared__ __align__(16) uint8_t raw[];
  bf16* sk = reinterpret_cast<bf16*>(raw);
  bf16* sv2 = sk + kTileElems;  // two tiles, one being filled
  bf16* ks3 = sv2 + 2 * kTileElems;
  float* D = reinterpret_cast<float*>(ks3 + kTerms * kTileElems);  // [blocks][64]
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.z, h = blockIdx.y, k0 = blockIdx.x * kSlab;
  const int K = a.key_dim, V = a.value_dim, tiles = (V + kTileV - 1) / kTileV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, m0 = (warp >> 1) * 16, v0 = (warp & 1) * 32;
  int row0;
  const int rows = chunk_rows(a, c, &row0);
  const Workspace ws(a);
  const bf16* kp = reinterpret_cast<const bf16*>(a.k) + (int64_t)row0 * a.k_stride + (int64_t)h * K;
  const bf16* vp = reinterpret_cast<const bf16*>(a.v) + (int64_t)row0 * a.v_stride + (int64_t)h * V;
  float* U = ws.state + ((size_t)c * a.num_heads + h) * K * V;
  load_rows(sk, kp + k0, a.k_stride, rows, min(kSlab, K - k0));
  load_rows(sv2, vp, a.v_stride, rows, min(kTileV, V));
  mma::cp_commit();
  {
    const int n = tid & 63, b = tid >> 6;
    Decays d;
    d.load(a, row0, rows, b * kBlock, h * K + k0 + n, k0 + n < K);
    mma::cp_wait<0>();
    __syncthreads();
    D[b * 64 + n] = keys_to_block_end(d, sk, ks3, b * kBlock, n);
  }
  for (int tile = 0; tile < tiles; ++tile) {
    const int c0 = tile * kTileV;
    if (tile > 0) mma::cp_wait<0>();
    __syncthreads();  // this tile is there, and the one before it has been read
    const bf16* sv = sv2 + (tile & 1) * kTileElems;
    if (tile + 1 < tiles) {
      load_rows(sv2 + (~tile & 1) * kTileElems, vp + c0 + kTileV, a.v_stride, rows, min(kTileV, V - c0 - kTileV));
      mma::cp_commit();
    }
    if (tile == 0 && tid < 64 && k0 + tid < K) {
      float p = 1.f;
#pragma unroll
      for (int j = 0; j < kBlocks; ++j) p *= D[j * 64 + tid];
      ws.keysum[((size_t)c * a.num_heads + h) * K + k0 + tid] = p;
    }
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
    for (int j = 0; j < kBlocks; ++j) {
      if (j > 0) {
        const float d0 = D[j * 64 + m0 + (lane >> 2)], d1 = D[j * 64 + m0 + (lane >> 2) + 8];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          acc[i][0] *= d0, acc[i][1] *= d0;
          acc[i][2] *= d1, acc[i][3] *= d1;
        }
      }
      // A[m = key dim][k = row]: stored row by row, so the fragments come transposed
      uint32_t fa[kTerms][4];
      const int mat = lane >> 3, krow = j * kBlock + ((mat >> 1) ? 8 : 0) + (lane & 7), kcol = m0 + ((mat & 1) ? 8 : 0);
#pragma unroll
      for (int t = 0; t < kTerms; ++t) mma::ldsm4t(fa[t], &ks3[t * kTileElems + krow * kPad + kcol]);
#pragma unroll
      for (int n2 = 0; n2 < 2; ++n2) {
        uint32_t fb[4];
        mma::ldsm4t(fb, &sv[(j * kBlock + (lane & 15)) * kPad + v0 + n2 * 16 + (lane >> 4) * 8]);
#pragma unroll
        for (int t = 0; t < kTerms; ++t) {
          mma::mma16816(acc[2 * n2], fa[t], fb[0], fb[1]);
          mma::mma16816(acc[2 * n2 + 1], fa[t], fb[2], fb[3]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int col = c0 + v0 + i * 8 + (lane & 3) * 2;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int kd = k0 + m0 + (lane >> 2) + half * 8;
        if (kd < K && col < V)
          *reinterpret_cast<float2*>(U + (size_t)kd * V + col) = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
      }
    }
  }
}

// ---- 3: outputs ------------------------------------------------------------------------------------------
// Two warps share a block: each takes half of a slab's key channels through all the products -- they are linear in the scores --
// and the two halves of the outputs meet at the end.
// sr sk sv | K's terms | { R, decays } fp32, over which the state on entry goes later (its three terms) | D, bonus, scores
constexpr int kBig = 2 * kFloatTile * 4;
constexpr int kScorePitch = kBlock + 1, kSwapPitch = 36;
static_assert(kBig >= kTerms * kTileElems * 2, "the state's terms go over R and the decays");
static_assert(kBig >= 2 * kBlocks * kBlock * kSwapPitch * 4, "so do the halves of the outputs");
constexpr int kOutputSmem =
    (3 + kTerms) * kTileElems * 2 + kBig + (kBlocks * 64 + 64) * 4 + 2 * kBlocks * kBlock * kScorePitch * 4;

__global__ void __launch_bounds__(kThreads, 2)
output_kernel(const b200_recurrence_args a) {
  extern __shared__ __align__(16) uint8_t raw[];
  bf16* sr = reinterpret_cast<bf16*>(raw);
  bf16* sk = sr + kTileElems;
  bf16* sv = sk + kTileElems;
  bf16* ks3 = sv + kTileElems;
  float* sR = reinterpret_cast<float*>(ks3 + kTerms * kTileElems);
  float* sw = sR + kFloatTile;
  bf16* ss = reinterpret_cast<bf16*>(sR);
  float* D = sw + kFloatTile;
  float* su = D + kBlocks * 64;
  float* own = su + 64;  // [warp][16 rows t][17]: scores inside the block, from the warp's channels
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.z, h = blockIdx.y, tile = blockIdx.x;
  const int K = a.key_dim, V = a.value_dim, c0 = tile * kTileV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int block = warp >> 1, half = warp & 1, base = block * kBlock;
  int row0;
  const int rows = chunk_rows(a, c, &row0);
  const Workspace ws(a);
  const bf16* rp = reinterpret_cast<const bf16*>(a.q) + (int64_t)row0 * a.q_stride + (int64_t)h * K;
  const bf16* kp = reinterpret_cast<const bf16*>(a.k) + (int64_t)row0 * a.k_stride + (int64_t)h * K;
  const bf16* vp = reinterpret_cast<const bf16*>(a.v) + (int64_t)row0 * a.v_stride + (int64_t)h * V + c0;
  const float* S = ws.state + ((size_t)c * a.num_heads + h) * K * V;
  load_rows(sv, vp, a.v_stride, rows, min(kTileV, V - c0));
  float* mine = own + warp * kBlock * kScorePitch;
  float sc[2 * (kBlocks - 1)][4], o[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[i][e] = 0.f;
#pragma unroll
  for (int i = 0; i < 2 * (kBlocks - 1); ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) sc[i][e] = 0.f;
  for (int k0 = 0; k0 < K; k0 += kSlab) {
    load_rows(sr, rp + k0, a.q_stride, rows, min(kSlab, K - k0));
    load_rows(sk, kp + k0, a.k_stride, rows, min(kSlab, K - k0));
    mma::cp_commit();
    float4 sx[4];  // the slab's state on entry, for later
    {
      const int n = tid & 63, b = tid >> 6, first = b * kBlock;
      if (tid < 64) su[tid] = k0 + tid < K ? a.skip[h * K + k0 + tid] : 0.f;
      Decays d;
      d.load(a, row0, rows, first, h * K + k0 + n, k0 + n < K);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = (tid >> 4) + i * 16, cc = (tid & 15) * 4;
        sx[i] = k0 + r < K && c0 + cc < V ? *reinterpret_cast<const float4*>(S + (size_t)(k0 + r) * V + c0 + cc)
                                          : make_float4(0.f, 0.f, 0.f, 0.f);
      }
      mma::cp_wait<0>();
      __syncthreads();
      float run = 1.f;
#pragma unroll
      for (int i = 0; i < kBlock; ++i) {
        sR[(first + i) * kPitch + n] = to_float(sr[(first + i) * kPad + n]) * run;
        sw[(first + i) * kPitch + n] = d.w[i];
        run *= d.w[i];
      }
      D[b * 64 + n] = keys_to_block_end(d, sk, ks3, first, n);
    }
    __syncthreads();
    // R of the block's rows and the warp's channels, as fragments: [k step][row half + column half][pair]
    float R[2][4][2];
#pragma unroll
    for (int ks = 0; ks < 2; ++ks)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float2 x = *reinterpret_cast<const float2*>(&sR[(base + g + (q & 1) * 8) * kPitch + half * 32 + ks * 16 + (q >> 1) * 8 + 2 * tq]);
        R[ks][q][0] = x.x, R[ks][q][1] = x.y;
      }
    {  // scores inside the block: lane = row s, 16 of the warp's channels
      const int s = lane & 15, n0 = half * 32 + (lane >> 4) * 16;
      float q[16];
#pragma unroll
      for (int i = 0; i < 16; i += 8) {
        const uint4 x4 = *reinterpret_cast<const uint4*>(&sk[(base + s) * kPad + n0 + i]);
        const bf16* x = reinterpret_cast<const bf16*>(&x4);
#pragma unroll
        for (int e = 0; e < 8; ++e) q[i + e] = to_float(x[e]);
      }
      float bonus = 0.f;  // the current row against itself
#pragma unroll
      for (int i = 0; i < 16; i += 8) {
        const uint4 x4 = *reinterpret_cast<const uint4*>(&sr[(base + s) * kPad + n0 + i]);
        const bf16* x = reinterpret_cast<const bf16*>(&x4);
#pragma unroll
        for (int e = 0; e < 8; ++e) bonus = fmaf(to_float(x[e]) * su[n0 + i + e], q[i + e], bonus);
      }
      bonus += __shfl_xor_sync(0xffffffffu, bonus, 16);
      if (lane < 16) mine[s * kScorePitch + s] = (k0 > 0 ? mine[s * kScorePitch + s] : 0.f) + bonus;
#pragma unroll 3
      for (int t = 1; t < kBlock; ++t) {
        float dot[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < 16; i += 8) {
          const uint4 x4 = *reinterpret_cast<const uint4*>(&sr[(base + t) * kPad + n0 + i]);
          const bf16* x = reinterpret_cast<const bf16*>(&x4);
#pragma unroll
          for (int e = 0; e < 8; ++e) dot[e & 3] = fmaf(to_float(x[e]), q[i + e], dot[e & 3]);
        }
        float sum = (dot[0] + dot[1]) + (dot[2] + dot[3]);
        sum += __shfl_xor_sync(0xffffffffu, sum, 16);
        if (lane < 16 && s < t) mine[t * kScorePitch + s] = (k0 > 0 ? mine[t * kScorePitch + s] : 0.f) + sum;
#pragma unroll
        for (int i = 0; i < 16; i += 4) {  // a row's own key does not decay before the row after the next reads it
          const float4 w = *reinterpret_cast<const float4*>(&sw[(base + t) * kPitch + n0 + i]);
          q[i] *= s < t ? w.x : 1.f, q[i + 1] *= s < t ? w.y : 1.f, q[i + 2] *= s < t ? w.z : 1.f, q[i + 3] *= s < t ? w.w : 1.f;
        }
      }
    }
    // against earlier blocks, nearest first; R picks up a block's decay after it
    auto split = [&](int ks, uint32_t (&fa)[kTerms][4]) {
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        uint32_t t[kTerms];
        mma::split_pair<kTerms>(R[ks][q][0], R[ks][q][1], t);
#pragma unroll
        for (int j = 0; j < kTerms; ++j) fa[j][q] = t[j];
      }
    };
#pragma unroll
    for (int j = kBlocks - 2; j >= 0; --j) {
      if (j >= block) continue;
#pragma unroll
      for (int ks = 0; ks < 2; ++ks) {
        const int col = half * 32 + ks * 16;
        uint32_t fa[kTerms][4];
        split(ks, fa);
#pragma unroll
        for (int y = 0; y < kTerms; ++y) {
          uint32_t fb[4];
          mma::ldsm4(fb, &ks3[y * kTileElems + (j * kBlock + (lane >> 4) * 8 + (lane & 7)) * kPad + col + ((lane >> 3) & 1) * 8]);
#pragma unroll
          for (int x = 0; x + y < kTerms; ++x) {
            mma::mma16816(sc[2 * j], fa[x], fb[0], fb[1]);
            mma::mma16816(sc[2 * j + 1], fa[x], fb[2], fb[3]);
          }
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float2 d = *reinterpret_cast<const float2*>(&D[j * 64 + col + (q >> 1) * 8 + 2 * tq]);
          R[ks][q][0] *= d.x, R[ks][q][1] *= d.y;
        }
      }
    }
    __syncthreads();  // R and the decays have been read everywhere: the state on entry goes over them
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (tid >> 4) + i * 16, cc = (tid & 15) * 4;
      uint32_t t0[kTerms], t1[kTerms];
      mma::split_pair<kTerms>(sx[i].x, sx[i].y, t0);
      mma::split_pair<kTerms>(sx[i].z, sx[i].w, t1);
#pragma unroll
      for (int j = 0; j < kTerms; ++j) *reinterpret_cast<uint2*>(&ss[j * kTileElems + r * kPad + cc]) = make_uint2(t0[j], t1[j]);
    }
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < 2; ++ks) {
      uint32_t fa[kTerms][4];
      split(ks, fa);
#pragma unroll
      for (int n2 = 0; n2 < 4; ++n2)
#pragma unroll
        for (int y = 0; y < kTerms; ++y) {
          uint32_t fb[4];
          mma::ldsm4t(fb, &ss[y * kTileElems + (half * 32 + ks * 16 + (lane & 15)) * kPad + n2 * 16 + (lane >> 4) * 8]);
#pragma unroll
          for (int x = 0; x + y < kTerms; ++x) {
            mma::mma16816(o[2 * n2], fa[x], fb[0], fb[1]);
            mma::mma16816(o[2 * n2 + 1], fa[x], fb[2], fb[3]);
          }
        }
    }
    __syncthreads();
  }
  // the scores' share of the outputs; those of the block itself on and below the diagonal
  auto values = [&](int j, const float (&lo)[4], const float (&hi)[4]) {  // scores of columns 0..7 and 8..15 of block j
    uint32_t p[4][kTerms];
    mma::split_pair<kTerms>(lo[0], lo[1], p[0]);
    mma::split_pair<kTerms>(lo[2], lo[3], p[1]);
    mma::split_pair<kTerms>(hi[0], hi[1], p[2]);
    mma::split_pair<kTerms>(hi[2], hi[3], p[3]);
#pragma unroll
    for (int n2 = 0; n2 < 4; ++n2) {
      uint32_t fb[4];
      mma::ldsm4t(fb, &sv[(j * kBlock + (lane & 15)) * kPad + n2 * 16 + (lane >> 4) * 8]);
#pragma unroll
      for (int x = 0; x < kTerms; ++x) {
        const uint32_t fa[4] = {p[0][x], p[1][x], p[2][x], p[3][x]};
        mma::mma16816(o[2 * n2], fa, fb[0], fb[1]);
        mma::mma16816(o[2 * n2 + 1], fa, fb[2], fb[3]);
      }
    }
  };
#pragma unroll
  for (int j = 0; j < kBlocks - 1; ++j)
    if (j < block) values(j, sc[2 * j], sc[2 * j + 1]);
  float dg[2][4];
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = g + (e >> 1) * 8, s = i * 8 + 2 * tq + (e & 1);
      dg[i][e] = s <= t ? mine[t * kScorePitch + s] : 0.f;
    }
  values(block, dg[0], dg[1]);
  // a warp leaves its partner the 32 columns that it does not store
  float* swap = sR + warp * kBlock * kSwapPitch;
  const float* other = sR + (warp ^ 1) * kBlock * kSwapPitch;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int cc = i * 8 + 2 * tq;
    float2 lo, hi;
    lo.x = half ? o[i][0] : o[i + 4][0], lo.y = half ? o[i][1] : o[i + 4][1];
    hi.x = half ? o[i][2] : o[i + 4][2], hi.y = half ? o[i][3] : o[i + 4][3];
    *reinterpret_cast<float2*>(&swap[g * kSwapPitch + cc]) = lo;
    *reinterpret_cast<float2*>(&swap[(g + 8) * kSwapPitch + cc]) = hi;
  }
  __syncthreads();
  bf16* out = reinterpret_cast<bf16*>(a.out);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int cc = i * 8 + 2 * tq, col = half * 32 + cc;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = base + g + e * 8;
      if (t >= rows || c0 + col >= V) continue;
      const float2 x = *reinterpret_cast<const float2*>(&other[(g + e * 8) * kSwapPitch + cc]);
      const float y0 = half ? o[i + 4][2 * e] : o[i][2 * e], y1 = half ? o[i + 4][2 * e + 1] : o[i][2 * e + 1];
      *reinterpret_cast<__nv_bfloat162*>(out + (int64_t)(row0 + t) * a.out_stride + (int64_t)h * V + c0 + col) =
          __floats2bfloat162_rn(y0 + x.x, y1 + x.y);
    }
  }
}

inline int launch(const b200_recurrence_args& a, cudaStream_t st) {
  B200_CHECK_ARG(a.workspace && a.workspace_bytes >= Workspace::bytes(a), "recurrence: workspace too small");
  B200_CHECK_ARG(a.chunk_seq && a.chunk_row && a.seq_chunk0, "recurrence: no chunk list");
  B200_CHECK_ARG(a.num_chunks <= 65535, "recurrence: more than 65535 chunks");
  static bool attr = false;
  if (!attr) {
    B200_CUDA_OK(cudaFuncSetAttribute(state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kStateSmem));
    B200_CUDA_OK(cudaFuncSetAttribute(output_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kOutputSmem));
    attr = true;
  }
  const dim3 grid((a.value_dim + kTileV - 1) / kTileV, a.num_heads, a.num_chunks);
  const dim3 slabs((a.key_dim + kSlab - 1) / kSlab, a.num_heads, a.num_chunks);
  B200_CUDA_OK(launch_pdl(state_kernel, slabs, dim3(kThreads), kStateSmem, st, a));
  const int blocks = (a.key_dim * a.value_dim / 4 + kScanThreads - 1) / kScanThreads;
  B200_CUDA_OK(launch_pdl(chunk_scan_kernel<kWkv>, dim3(blocks, a.num_heads, a.num_seqs), dim3(kScanThreads), 0, st, a, blocks));
  B200_CUDA_OK(launch_pdl(output_kernel, grid, dim3(kThreads), kOutputSmem, st, a));
  return check_launch("recurrence (decays per key channel)");
}

}  // namespace wkv
}  // namespace rec
}  // namespace b200
