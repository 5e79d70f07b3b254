// Chunked form of the gated linear recurrence on tensor cores.  With cumulative log decays inside a 64-row chunk,
//   out_t = scale_t (S_in^T q_t) + sum_{s <= t} weight_ts (q_t . k_s) v_s,   S_out = keep S_in + sum_s w_s k_s v_s^T,
// so all chunks of all segments run at once in three launches:
//   1. chunk_state_kernel   every chunk's own contribution U = sum_s w_s k_s v_s^T  -> workspace (fp32)
//   2. chunk_scan_kernel    per state element, over the chunks of a segment: S_in replaces U in place, slot updated
//   3. chunk_output_kernel  the outputs from S_in and the chunk's own rows
// q, k, v are bf16 as the projections left them; every 32-bit factor (state, decay weights times scores) enters the
// 16-bit products as an exact three-term bf16 split, so the recurrence keeps 24 significant bits.
#pragma once

#include "mma_sync.cuh"
#include "recurrence_common.cuh"

namespace b200 {
namespace rec {

using bf16 = __nv_bfloat16;
constexpr int kChunk = B200_RECURRENCE_CHUNK;
constexpr int kSlab = 64;   // key dimensions per pass
constexpr int kPad = 72;    // shared row pitch (bf16): ldmatrix without bank conflicts
constexpr int kTerms = 3;
constexpr int kTileElems = 64 * kPad;

// workspace: U / S_in [chunks][heads][K][V], then per (chunk, head): key-sum (kind 3: decay over the chunk) [K], then {total, amax, m_in, first_m}
struct Workspace {
  float *state, *keysum, *scal, *gates;  // gates (128-row form): per (chunk, head) {cum, src, top, weight}[128]
  __host__ __device__ Workspace(const b200_recurrence_args& a) {
    const size_t ch = (size_t)a.num_chunks * a.num_heads;
    state = reinterpret_cast<float*>(a.workspace);
    keysum = state + ch * a.key_dim * a.value_dim;
    scal = keysum + (a.kind == kMlstm || a.kind == kWkv ? ch * a.key_dim : 0);
    gates = scal + 4 * ch;
  }
  static size_t bytes(const b200_recurrence_args& a) {
    const size_t ch = (size_t)a.num_chunks * a.num_heads;
    return (ch * a.key_dim * a.value_dim + (a.kind == kMlstm || a.kind == kWkv ? ch * a.key_dim : 0) + 4 * ch +
            (a.chunk == B200_RECURRENCE_CHUNK_TC ? ch * 4 * B200_RECURRENCE_CHUNK_TC : 0)) * sizeof(float);
  }
};

// The gates of a chunk's ROWS rows.  cum[t]: cumulative log decay; SSD: src[t] = step size dt (lightning: 1), mLSTM: src[t] = log input
// weight minus cum[t], top[t] = running maximum of src.  Rows past the end contribute nothing.  All threads call.
template <int KIND, int ROWS = kChunk>
__device__ __forceinline__ void chunk_gates(const b200_recurrence_args& a, int row0, int rows, int h, float* cum,
                                            float* src, float* top) {
  const int tid = threadIdx.x;
  constexpr int E = ROWS / 32;
  if (tid < ROWS) {
    float decay = 0.f, in = KIND == kMlstm ? -INFINITY : 0.f;
    if (tid < rows && KIND == kLightning) {
      in = 1.f;
      decay = -a.rate[h];
    } else if (tid < rows) {
      const int64_t off = (int64_t)(row0 + tid) * a.gate_stride + h;
      const float ga = to_float(reinterpret_cast<const bf16*>(a.gate_a)[off]);
      if (KIND == kSsd) {
        in = softplus_f(ga + a.bias_a[h]);
        decay = -a.rate[h] * in;
      } else {
        const float gb = to_float(reinterpret_cast<const bf16*>(a.gate_b)[off]);
        in = a.gate_cap * tanhf((ga + a.bias_a[h]) / a.gate_cap);
        decay = -softplus_f(-a.gate_cap * tanhf((gb + a.bias_b[h]) / a.gate_cap));
      }
    }
    cum[tid] = decay;
    src[tid] = in;
  }
  __syncthreads();
  if (tid < 32) {
    float x[E], run = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e) {
      run += cum[E * tid + e];
      x[e] = run;
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float y = __shfl_up_sync(0xffffffffu, run, o);
      if (tid >= o) run += y;
    }
    float excl = __shfl_up_sync(0xffffffffu, run, 1);
    if (tid == 0) excl = 0.f;
#pragma unroll
    for (int e = 0; e < E; ++e) cum[E * tid + e] = x[e] + excl;
    if (KIND == kMlstm) {
      float mx = -INFINITY, m[E];
#pragma unroll
      for (int e = 0; e < E; ++e) {
        const float v = src[E * tid + e] - (x[e] + excl);
        src[E * tid + e] = v;
        mx = fmaxf(mx, v);
        m[e] = mx;
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, mx, o);
        if (tid >= o) mx = fmaxf(mx, y);
      }
      float below = __shfl_up_sync(0xffffffffu, mx, 1);
      if (tid == 0) below = -INFINITY;
#pragma unroll
      for (int e = 0; e < E; ++e) top[E * tid + e] = fmaxf(below, m[e]);
    }
  }
  __syncthreads();
}

// rows x 64 columns (first column c0, `cols` valid) of a bf16 matrix into a padded tile, zeros elsewhere.
__device__ __forceinline__ void load_tile(bf16* dst, const bf16* src, int64_t stride, int rows, int cols) {
  for (int i = threadIdx.x; i < 64 * 8; i += 128) {
    const int r = i >> 3, c = (i & 7) * 8;
    const bool live = r < rows && c < cols;
    mma::cp_async16(dst + r * kPad + c, live ? src + (int64_t)r * stride + c : src, live);
  }
}

__device__ __forceinline__ int chunk_rows(const b200_recurrence_args& a, int c, int* row0) {
  const int s = a.chunk_seq[c];
  *row0 = a.chunk_row[c];
  return min(a.chunk, a.cu_seqlens[s + 1] - *row0);
}

// ---- 1: the chunk's own contribution -----------------------------------------------------------
template <int KIND>
__global__ void __launch_bounds__(128)
chunk_state_kernel(const b200_recurrence_args a) {
  __shared__ __align__(16) bf16 sk[kTileElems];
  __shared__ __align__(16) bf16 sv[kTerms][kTileElems];
  __shared__ float cum[kChunk], src[kChunk], top[kChunk], wgt[kChunk];
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.z, h = blockIdx.y, tile = blockIdx.x;
  const int K = a.key_dim, V = a.value_dim, c0 = tile * kTileV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = h / (a.num_heads / a.num_groups);
  int row0;
  const int rows = chunk_rows(a, c, &row0);
  const Workspace ws(a);
  const bf16* kp = reinterpret_cast<const bf16*>(a.k) + (int64_t)row0 * a.k_stride + (int64_t)g * K;
  const bf16* vp = reinterpret_cast<const bf16*>(a.v) + (int64_t)row0 * a.v_stride + (int64_t)h * V + c0;
  load_tile(sk, kp, a.k_stride, rows, min(kSlab, K));
  mma::cp_commit();
  chunk_gates<KIND>(a, row0, rows, h, cum, src, top);
  const float total = cum[kChunk - 1];  // rows past the end add no decay
  if (tid < kChunk) {
    float w = 0.f;
    if (tid < rows) w = KIND != kMlstm ? src[tid] * expf(total - cum[tid]) : expf(src[tid] - top[kChunk - 1]);
    wgt[tid] = w;
  }
  __syncthreads();
  // weighted values, split: the products below then have exact 16-bit operands
  for (int i = tid; i < 64 * 32; i += 128) {
    const int r = i >> 5, cc = (i & 31) * 2;
    float x = 0.f, y = 0.f;
    if (r < rows) {
      const bf16* vr = vp + (int64_t)r * a.v_stride;
      if (c0 + cc < V) x = wgt[r] * to_float(vr[cc]);
      if (c0 + cc + 1 < V) y = wgt[r] * to_float(vr[cc + 1]);
    }
    uint32_t t[kTerms];
    mma::split_pair<kTerms>(x, y, t);
#pragma unroll
    for (int j = 0; j < kTerms; ++j) *reinterpret_cast<uint32_t*>(&sv[j][r * kPad + cc]) = t[j];
  }
  float* U = ws.state + ((size_t)c * a.num_heads + h) * K * V;
  float* scal = ws.scal + 4 * ((size_t)c * a.num_heads + h);
  if (tile == 0 && tid == 0) {
    scal[0] = total;
    if (KIND == kMlstm) {
      scal[1] = top[kChunk - 1];
      const int s = a.chunk_seq[c];
      if (row0 == a.cu_seqlens[s]) {
        const int tiles = gridDim.x;
        const bool fresh = a.seq_lens[s] == a.cu_seqlens[s + 1] - row0;
        scal[2] = fresh ? 0.f : a.max_state[((int64_t)a.slots[s] * a.num_heads + h) * tiles];
      }
    }
  }
  for (int k0 = 0; k0 < K; k0 += kSlab) {
    mma::cp_wait<0>();
    __syncthreads();
    float acc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      // A[m = key dim][k = row]: the tile is stored row-major by row, so the fragments come transposed
      uint32_t fa[4];
      {
        const int mat = lane >> 3, rr = lane & 7;
        const int krow = ks * 16 + ((mat >> 1) ? 8 : 0) + rr, kcol = warp * 16 + ((mat & 1) ? 8 : 0);
        mma::ldsm4t(fa, &sk[krow * kPad + kcol]);
      }
#pragma unroll
      for (int n2 = 0; n2 < 4; ++n2) {
#pragma unroll
        for (int j = 0; j < kTerms; ++j) {
          uint32_t fb[4];
          mma::ldsm4t(fb, &sv[j][(ks * 16 + (lane & 15)) * kPad + n2 * 16 + (lane >> 4) * 8]);
          mma::mma16816(acc[2 * n2], fa, fb[0], fb[1]);
          mma::mma16816(acc[2 * n2 + 1], fa, fb[2], fb[3]);
        }
      }
    }
    if (KIND == kMlstm && tile == 0 && tid < kSlab && k0 + tid < K) {
      float n = 0.f;
      for (int r = 0; r < rows; ++r) n += wgt[r] * to_float(sk[r * kPad + tid]);
      ws.keysum[((size_t)c * a.num_heads + h) * K + k0 + tid] = n;
    }
    __syncthreads();
    if (k0 + kSlab < K) {
      load_tile(sk, kp + k0 + kSlab, a.k_stride, rows, min(kSlab, K - k0 - kSlab));
      mma::cp_commit();
    }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int col = c0 + n * 8 + (lane & 3) * 2;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int kd = k0 + warp * 16 + (lane >> 2) + half * 8;
        if (kd < K && col < V)
          *reinterpret_cast<float2*>(U + (size_t)kd * V + col) = make_float2(acc[n][2 * half], acc[n][2 * half + 1]);
      }
    }
  }
}

// ---- 2: the scan over a segment's chunks -----------------------------------------------------
// blockIdx.x < state blocks: 4 state elements a thread; the last block (mLSTM): the normaliser and the maximum.
constexpr int kScanThreads = 128;
template <int KIND>
__global__ void __launch_bounds__(kScanThreads)
chunk_scan_kernel(const b200_recurrence_args a, int state_blocks) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.z, h = blockIdx.y;
  const int len = a.cu_seqlens[s + 1] - a.cu_seqlens[s];
  if (len <= a.seq_limit) return;
  const int nc = (len + a.chunk - 1) / a.chunk, cfirst = a.seq_chunk0[s];
  const bool fresh = a.seq_lens[s] == len;
  const int K = a.key_dim, V = a.value_dim;
  const Workspace ws(a);
  const int64_t slot_head = (int64_t)a.slots[s] * a.num_heads + h;
  const float* scal = ws.scal + 4 * ((size_t)cfirst * a.num_heads + h);
  const size_t sstep = 4 * (size_t)a.num_heads;
  if ((int)blockIdx.x < state_blocks) {
    const size_t i = ((size_t)blockIdx.x * kScanThreads + threadIdx.x) * 4;
    if (i >= (size_t)K * V) return;
    float4* st = reinterpret_cast<float4*>(a.state + slot_head * (int64_t)K * V + i);
    float* u = ws.state + ((size_t)cfirst * a.num_heads + h) * K * V + i;
    const size_t ustep = (size_t)a.num_heads * K * V;
    float4 S = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *st;
    float m = KIND == kMlstm ? scal[2] : 0.f;
    constexpr int AHEAD = KIND == kWkv ? 8 : 4;
    float4 buf[AHEAD];
    float kept[KIND == kWkv ? AHEAD : 1];  // decay of this key row over a chunk
    const float* kp = ws.keysum + ((size_t)cfirst * a.num_heads + h) * K + (KIND == kWkv ? i / V : 0);
    const size_t kstep = (size_t)a.num_heads * K;
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
      if (j < nc) {
        buf[j] = *reinterpret_cast<const float4*>(u + j * ustep);
        if (KIND == kWkv) kept[KIND == kWkv ? j : 0] = kp[j * kstep];
      }
    for (int c0 = 0; c0 < nc; c0 += AHEAD) {
#pragma unroll
      for (int j = 0; j < AHEAD; ++j) {
        const int c = c0 + j;
        if (c >= nc) break;
        const float4 U = buf[j];
        float keep = KIND == kWkv ? kept[KIND == kWkv ? j : 0] : 0.f, add = 1.f;
        if (c + AHEAD < nc) {
          buf[j] = *reinterpret_cast<const float4*>(u + (size_t)(c + AHEAD) * ustep);
          if (KIND == kWkv) kept[KIND == kWkv ? j : 0] = kp[(c + AHEAD) * kstep];
        }
        *reinterpret_cast<float4*>(u + (size_t)c * ustep) = S;
        if (KIND == kWkv) {
        } else if (KIND != kMlstm) {
          keep = expf(scal[c * sstep]);
        } else {
          const float amax = scal[c * sstep + 1], b = fmaxf(m, amax);
          keep = expf(m - b);
          add = expf(amax - b);
          m = scal[c * sstep] + b;
        }
        S.x = keep * S.x + add * U.x;
        S.y = keep * S.y + add * U.y;
        S.z = keep * S.z + add * U.z;
        S.w = keep * S.w + add * U.w;
      }
    }
    *st = S;
  } else if (KIND == kMlstm) {
    const int tiles = (V + kTileV - 1) / kTileV;
    float* keys = ws.keysum + ((size_t)cfirst * a.num_heads + h) * K;
    float* sc = const_cast<float*>(scal);
    const size_t kstep = (size_t)a.num_heads * K;
    float* N = a.norm_state + slot_head * tiles * (int64_t)K;
    const float m0 = scal[2];
    float m = m0;
    for (int k0 = 0; k0 < K; k0 += kScanThreads) {
      const int k = k0 + threadIdx.x;
      m = m0;
      float n = (fresh || k >= K) ? 0.f : N[k];
      for (int c = 0; c < nc; ++c) {
        const float amax = sc[c * sstep + 1], b = fmaxf(m, amax);
        if (k < K) {
          const float u = keys[c * kstep + k];
          keys[c * kstep + k] = n;
          n = expf(m - b) * n + expf(amax - b) * u;
        }
        if (k == 0) sc[c * sstep + 3] = m;  // the maximum on entry to the chunk ([2] is only read here and above)
        m = sc[c * sstep] + b;
      }
      if (k < K)
        for (int t = 0; t < tiles; ++t) N[(int64_t)t * K + k] = n;
    }
    if (threadIdx.x < tiles) a.max_state[slot_head * tiles + threadIdx.x] = m;
    for (int t = threadIdx.x + kScanThreads; t < tiles; t += kScanThreads) a.max_state[slot_head * tiles + t] = m;
  }
}

// ---- 3: outputs -----------------------------------------------------------------------------------
constexpr int kOutSmem = (3 + kTerms) * kTileElems * 2 + (6 * 64 + 64) * 4;
template <int KIND>
__global__ void __launch_bounds__(128)
chunk_output_kernel(const b200_recurrence_args a) {
  extern __shared__ __align__(16) uint8_t raw[];
  bf16* sq = reinterpret_cast<bf16*>(raw);
  bf16* sk = sq + kTileElems;
  bf16* sv = sk + kTileElems;
  bf16* ss = sv + kTileElems;  // kTerms tiles: the state on entry, split
  float* cum = reinterpret_cast<float*>(ss + kTerms * kTileElems);
  float *src = cum + 64, *top = src + 64, *scale = top + 64, *dots = scale + 64, *nin = dots + 128;
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.z, h = blockIdx.y, tile = blockIdx.x;
  const int K = a.key_dim, V = a.value_dim, c0 = tile * kTileV;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = h / (a.num_heads / a.num_groups);
  int row0;
  const int rows = chunk_rows(a, c, &row0);
  const Workspace ws(a);
  const bf16* qp = reinterpret_cast<const bf16*>(a.q) + (int64_t)row0 * a.q_stride + (int64_t)g * K;
  const bf16* kp = reinterpret_cast<const bf16*>(a.k) + (int64_t)row0 * a.k_stride + (int64_t)g * K;
  const bf16* vp = reinterpret_cast<const bf16*>(a.v) + (int64_t)row0 * a.v_stride + (int64_t)h * V + c0;
  const float* S = ws.state + ((size_t)c * a.num_heads + h) * K * V;
  const float* keysum = ws.keysum + ((size_t)c * a.num_heads + h) * K;
  load_tile(sv, vp, a.v_stride, rows, min(kTileV, V - c0));
  float sc[8][4], o[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) sc[n][e] = o[n][e] = 0.f;
  float dot = 0.f;  // mLSTM: q . normaliser-on-entry; row tid / 2, half of the slab each
  for (int k0 = 0; k0 < K; k0 += kSlab) {
    load_tile(sq, qp + k0, a.q_stride, rows, min(kSlab, K - k0));
    load_tile(sk, kp + k0, a.k_stride, rows, min(kSlab, K - k0));
    mma::cp_commit();
    for (int i = tid; i < 64 * 16; i += 128) {
      const int r = i >> 4, cc = (i & 15) * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (k0 + r < K && c0 + cc < V) x = *reinterpret_cast<const float4*>(S + (size_t)(k0 + r) * V + c0 + cc);
      uint32_t t0[kTerms], t1[kTerms];
      mma::split_pair<kTerms>(x.x, x.y, t0);
      mma::split_pair<kTerms>(x.z, x.w, t1);
#pragma unroll
      for (int j = 0; j < kTerms; ++j)
        *reinterpret_cast<uint2*>(&ss[j * kTileElems + r * kPad + cc]) = make_uint2(t0[j], t1[j]);
    }
    if (KIND == kMlstm && tid < kSlab) nin[tid] = k0 + tid < K ? keysum[k0 + tid] : 0.f;
    mma::cp_wait<0>();
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t fa[4];
      mma::ldsm4(fa, &sq[(warp * 16 + (lane & 15)) * kPad + ks * 16 + (lane >> 4) * 8]);
#pragma unroll
      for (int n2 = 0; n2 < 4; ++n2) {
        if (n2 <= warp) {  // scores above the diagonal are not needed
          uint32_t fb[4];
          mma::ldsm4(fb, &sk[(n2 * 16 + (lane >> 4) * 8 + (lane & 7)) * kPad + ks * 16 + ((lane >> 3) & 1) * 8]);
          mma::mma16816(sc[2 * n2], fa, fb[0], fb[1]);
          mma::mma16816(sc[2 * n2 + 1], fa, fb[2], fb[3]);
        }
#pragma unroll
        for (int j = 0; j < kTerms; ++j) {
          uint32_t fb[4];
          mma::ldsm4t(fb, &ss[j * kTileElems + (ks * 16 + (lane & 15)) * kPad + n2 * 16 + (lane >> 4) * 8]);
          mma::mma16816(o[2 * n2], fa, fb[0], fb[1]);
          mma::mma16816(o[2 * n2 + 1], fa, fb[2], fb[3]);
        }
      }
    }
    if (KIND == kMlstm) {
      const bf16* qr = &sq[(tid >> 1) * kPad + (tid & 1) * 32];
#pragma unroll 8
      for (int i = 0; i < 32; ++i) dot += to_float(qr[i]) * nin[(tid & 1) * 32 + i];
    }
    __syncthreads();
  }
  chunk_gates<KIND>(a, row0, rows, h, cum, src, top);
  const float m_in = KIND == kMlstm ? ws.scal[4 * ((size_t)c * a.num_heads + h) + 3] : 0.f;
  if (KIND == kMlstm) {
    dots[tid] = dot;
    if (tid < kChunk) top[tid] = fmaxf(m_in, top[tid]);  // the running maximum minus cum
  }
  if (tid < kChunk) scale[tid] = KIND != kMlstm ? expf(cum[tid]) : expf(m_in - fmaxf(m_in, top[tid]));
  __syncthreads();
  float rowsum[2] = {0.f, 0.f};
#pragma unroll
  for (int n = 0; n < 8; ++n) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = warp * 16 + (lane >> 2) + (e >> 1) * 8, s = n * 8 + (lane & 3) * 2 + (e & 1);
      o[n][e] *= scale[t] * a.q_scale;
      float w = 0.f;
      if (s <= t && s < rows) w = KIND != kMlstm ? expf(cum[t] - cum[s]) * src[s] : expf(src[s] - top[t]);
      sc[n][e] *= w * a.q_scale;
      rowsum[e >> 1] += sc[n][e];
    }
  }
#pragma unroll
  for (int ks = 0; ks < 4; ++ks) {
    if (ks > warp) break;  // rows past this warp's own are masked
    uint32_t p[4][kTerms];
    mma::split_pair<kTerms>(sc[2 * ks][0], sc[2 * ks][1], p[0]);
    mma::split_pair<kTerms>(sc[2 * ks][2], sc[2 * ks][3], p[1]);
    mma::split_pair<kTerms>(sc[2 * ks + 1][0], sc[2 * ks + 1][1], p[2]);
    mma::split_pair<kTerms>(sc[2 * ks + 1][2], sc[2 * ks + 1][3], p[3]);
#pragma unroll
    for (int n2 = 0; n2 < 4; ++n2) {
      uint32_t fb[4];
      mma::ldsm4t(fb, &sv[(ks * 16 + (lane & 15)) * kPad + n2 * 16 + (lane >> 4) * 8]);
#pragma unroll
      for (int j = 0; j < kTerms; ++j) {
        const uint32_t fa[4] = {p[0][j], p[1][j], p[2][j], p[3][j]};
        mma::mma16816(o[2 * n2], fa, fb[0], fb[1]);
        mma::mma16816(o[2 * n2 + 1], fa, fb[2], fb[3]);
      }
    }
  }
  float div[2] = {1.f, 1.f};
  if (KIND == kMlstm) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      rowsum[e] += __shfl_xor_sync(0xffffffffu, rowsum[e], 1);
      rowsum[e] += __shfl_xor_sync(0xffffffffu, rowsum[e], 2);
      const int t = warp * 16 + (lane >> 2) + e * 8;
      const float dn = rowsum[e] + (dots[2 * t] + dots[2 * t + 1]) * scale[t] * a.q_scale;
      div[e] = 1.f / (fmaxf(fabsf(dn), expf(-(cum[t] + top[t]))) + 1e-6f);
    }
  }
  const float skip = KIND == kSsd ? a.skip[h] : 0.f;
  bf16* out = reinterpret_cast<bf16*>(a.out);
#pragma unroll
  for (int n = 0; n < 8; ++n) {
    const int cc = n * 8 + (lane & 3) * 2;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = warp * 16 + (lane >> 2) + e * 8;
      if (t >= rows || c0 + cc >= V) continue;
      float x = o[n][2 * e] * div[e], y = o[n][2 * e + 1] * div[e];
      if (KIND == kSsd) {
        x += skip * to_float(sv[t * kPad + cc]);
        y += skip * to_float(sv[t * kPad + cc + 1]);
      }
      *reinterpret_cast<__nv_bfloat162*>(out + (int64_t)(row0 + t) * a.out_stride + (int64_t)h * V + c0 + cc) =
          __floats2bfloat162_rn(x, y);
    }
  }
}

inline bool can_chunk(const b200_recurrence_args& a) {
  auto ok = [](const void* p, int64_t stride) { return ((uintptr_t)p & 15) == 0 && stride % 8 == 0; };
  return a.dtype == B200_BF16 && a.key_dim % 8 == 0 && a.value_dim % 8 == 0 && ok(a.q, a.q_stride) &&
         ok(a.k, a.k_stride) && ok(a.v, a.v_stride) && ((uintptr_t)a.out & 3) == 0 && a.out_stride % 2 == 0 &&
         ((uintptr_t)a.state & 15) == 0;
}

template <int KIND>
int launch_chunked(const b200_recurrence_args& a, cudaStream_t st) {
  B200_CHECK_ARG(a.workspace && a.workspace_bytes >= Workspace::bytes(a), "recurrence: workspace too small");
  B200_CHECK_ARG(a.chunk_seq && a.chunk_row && a.seq_chunk0, "recurrence: no chunk list");
  B200_CHECK_ARG(a.num_chunks <= 65535, "recurrence: more than 65535 chunks");
  const int tiles = (a.value_dim + kTileV - 1) / kTileV;
  const dim3 grid(tiles, a.num_heads, a.num_chunks);
  B200_CUDA_OK(launch_pdl(chunk_state_kernel<KIND>, grid, dim3(128), 0, st, a));
  const int blocks = (a.key_dim * a.value_dim / 4 + kScanThreads - 1) / kScanThreads;
  B200_CUDA_OK(launch_pdl(chunk_scan_kernel<KIND>, dim3(blocks + (KIND == kMlstm ? 1 : 0), a.num_heads, a.num_seqs),
                          dim3(kScanThreads), 0, st, a, blocks));
  static bool attr = false;  // per instantiation
  if (!attr) {
    B200_CUDA_OK(cudaFuncSetAttribute(chunk_output_kernel<KIND>, cudaFuncAttributeMaxDynamicSharedMemorySize, kOutSmem));
    attr = true;
  }
  B200_CUDA_OK(launch_pdl(chunk_output_kernel<KIND>, grid, dim3(128), kOutSmem, st, a));
  return check_launch("recurrence (chunked)");
}

}  // namespace rec
}  // namespace b200
