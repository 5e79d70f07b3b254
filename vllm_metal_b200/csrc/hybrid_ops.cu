// Norms, gates, activations and the short convolution around the mixers of hybrid decoders
// (include/b200_hybrid_ops.h).  HBM / launch bound: one read, one write, fp32 arithmetic.
#include "../../include/b200_hybrid_ops.h"
#include "common.cuh"

#include <type_traits>

namespace b200 {
namespace {

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float gelu_erf_f(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }
constexpr int kActGelu = 0, kActSilu = 1, kActTanh = 2, kActXielu = 3;
__device__ __forceinline__ float xielu_f(float z, float a, float b) {
  return z > 0.f ? fmaf(a * z, z, 0.5f * z) : fmaf(b, expm1f(z) - z, 0.5f * z);
}

template <int THREADS>
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  const float t = warp_sum(lane < THREADS / 32 ? red[lane] : 0.f);
  __syncthreads();
  return t;
}

// ---- embedding row -> fp32 stream ------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
embed_rows_kernel(const int32_t* __restrict__ ids, const T* __restrict__ table, float* __restrict__ out, int vocab,
                  int dim, int64_t out_stride) {
  pdl_trigger();
  pdl_wait();
  const int id = ids[blockIdx.x];
  float* o = out + (int64_t)blockIdx.x * out_stride;
  const bool ok = id >= 0 && id < vocab;
  for (int d = threadIdx.x; d < dim; d += 256) o[d] = ok ? to_float(table[(int64_t)id * dim + d]) : 0.f;
}

// ---- RMS norm of the fp32 stream ---------------------------------------------------------------
template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
stream_norm_kernel(const float* __restrict__ x, const int64_t* __restrict__ row_ids, const float* __restrict__ weight,
                   T* __restrict__ out, int dim, int64_t x_stride, int64_t out_stride, float eps, float offset) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  const int64_t row = row_ids ? row_ids[blockIdx.x] : blockIdx.x;
  const float* xr = x + row * x_stride;
  T* o = out + (int64_t)blockIdx.x * out_stride;
  float ss = 0.f;
  if (VEC) {
    constexpr int NR = 4;  // 4096 columns stay in registers, longer rows are read twice
    const int nv = dim >> 2;
    float4 keep[NR];
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int i = threadIdx.x + j * 256;
      keep[j] = i < nv ? reinterpret_cast<const float4*>(xr)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
      ss += keep[j].x * keep[j].x + keep[j].y * keep[j].y + keep[j].z * keep[j].z + keep[j].w * keep[j].w;
    }
    for (int i = threadIdx.x + NR * 256; i < nv; i += 256) {
      const float4 v = reinterpret_cast<const float4*>(xr)[i];
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float inv = 1.f / sqrtf(block_sum<256>(ss, red) / (float)dim + eps);
    auto put = [&](int i, float4 v) {
      const float4 w = reinterpret_cast<const float4*>(weight)[i];
      T r[4] = {from_float<T>(v.x * inv * (w.x + offset)), from_float<T>(v.y * inv * (w.y + offset)),
                from_float<T>(v.z * inv * (w.z + offset)), from_float<T>(v.w * inv * (w.w + offset))};
      if (sizeof(T) == 4)
        reinterpret_cast<uint4*>(o)[i] = *reinterpret_cast<uint4*>(r);
      else
        reinterpret_cast<uint2*>(o)[i] = *reinterpret_cast<uint2*>(r);
    };
#pragma unroll
    for (int j = 0; j < NR; ++j)
      if (threadIdx.x + j * 256 < nv) put(threadIdx.x + j * 256, keep[j]);
    for (int i = threadIdx.x + NR * 256; i < nv; i += 256) put(i, reinterpret_cast<const float4*>(xr)[i]);
  } else {
    for (int d = threadIdx.x; d < dim; d += 256) ss += xr[d] * xr[d];
    const float inv = 1.f / sqrtf(block_sum<256>(ss, red) / (float)dim + eps);
    for (int d = threadIdx.x; d < dim; d += 256) o[d] = from_float<T>(xr[d] * inv * (weight[d] + offset));
  }
}

// ---- gate -> group norm -> gate, and the feed-forward activation ----------------------------
// Roles by blockIdx.x: the first `norm_blocks` own groups of the mixer half (a warp or the whole CTA per group), the
// rest 1024 columns of the activation half each.
template <typename T, bool WARP_GROUPS>
__global__ void __launch_bounds__(256)
mixer_finish_kernel(const b200_mixer_finish_args a, int norm_blocks) {
  pdl_trigger();
  pdl_wait();
  const int64_t r = blockIdx.y;
  T* o = reinterpret_cast<T*>(a.out) + r * a.out_stride;
  if ((int)blockIdx.x < norm_blocks) {
    __shared__ float red[8];
    const T* y = reinterpret_cast<const T*>(a.y) + r * a.y_stride;
    const T* pre = a.pre_gate ? reinterpret_cast<const T*>(a.pre_gate) + r * a.pre_stride : nullptr;
    const T* post = a.post_gate ? reinterpret_cast<const T*>(a.post_gate) + r * a.post_stride : nullptr;
    const int gs = a.group_size > 0 ? a.group_size : 256;  // without a norm: slices of 256 columns
    const int group = WARP_GROUPS ? blockIdx.x * 8 + (threadIdx.x >> 5) : blockIdx.x;
    const int c0 = group * gs, c1 = min(c0 + gs, a.inner);
    constexpr int STEP = WARP_GROUPS ? 32 : 256;
    const int first = WARP_GROUPS ? (threadIdx.x & 31) : threadIdx.x;
    auto value = [&](int c) {
      const int yc = a.y_head_dim > 0 ? c / a.y_head_dim * a.y_head_stride + c % a.y_head_dim : c;
      float v = to_float(y[yc]);
      if (pre) {
        const float z = to_float(pre[c]);
        v *= z * sigmoid_f(z);
      }
      return v;
    };
    constexpr int KEEP = 8;
    float keep[KEEP];
    float ss = 0.f, inv = 1.f;
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      const int c = c0 + first + j * STEP;
      keep[j] = c < c1 ? value(c) : 0.f;
      ss += keep[j] * keep[j];
    }
    for (int c = c0 + first + KEEP * STEP; c < c1; c += STEP) {
      const float v = value(c);
      ss += v * v;
    }
    if (a.group_size > 0) {
      ss = WARP_GROUPS ? warp_sum(ss) : block_sum<256>(ss, red);
      inv = 1.f / sqrtf(ss / (float)gs + a.eps);
    }
    auto put = [&](int c, float v) {
      v *= inv;
      if (a.weight) v *= a.weight[c];
      if (post) {
        const float z = to_float(post[c]), g = sigmoid_f(z);
        v *= a.post_silu ? z * g : g;
      }
      o[c] = from_float<T>(v);
    };
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      const int c = c0 + first + j * STEP;
      if (c < c1) put(c, keep[j]);
    }
    for (int c = c0 + first + KEEP * STEP; c < c1; c += STEP) put(c, value(c));
  } else {
    const T* in = reinterpret_cast<const T*>(a.act_in) + r * a.act_stride;
    const T* mul = a.act_mul ? reinterpret_cast<const T*>(a.act_mul) + r * a.mul_stride : nullptr;
    const int base = ((int)blockIdx.x - norm_blocks) * 1024;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = base + j * 256 + threadIdx.x;
      if (i >= a.act_dim) continue;
      const float z = to_float(in[i]);
      const float v = a.act_kind == kActSilu   ? z * sigmoid_f(z)
                      : a.act_kind == kActGelu ? gelu_erf_f(z)
                      : a.act_kind == kActTanh ? tanhf(z)
                                               : xielu_f(z, a.act_a, a.act_b);
      o[a.act_offset + i] = from_float<T>(mul ? v * to_float(mul[i]) : v);
    }
  }
  // alignment padding: [inner, act_offset) and [act_offset + act_dim, out_cols)
  if (blockIdx.x == 0) {
    const int lo = a.act_dim > 0 ? a.act_offset : a.out_cols;
    for (int c = a.inner + threadIdx.x; c < lo; c += 256) o[c] = from_float<T>(0.f);
    if (a.act_dim > 0)
      for (int c = a.act_offset + a.act_dim + threadIdx.x; c < a.out_cols; c += 256) o[c] = from_float<T>(0.f);
  }
}

// The same for 16-bit types whose rows, groups and offsets are whole 16-byte units: 8 columns a thread and step, the
// group held in registers between its norm and its store.  LANES threads share a group, VPL units each; the activation
// half takes ACT units a thread.
template <typename T>
struct alignas(16) Vec8 {
  T e[8];
};
__device__ __forceinline__ float fast_sigmoid(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

// In 16-bit results: near zero the first terms of the series, where exp(z) - 1 - z would cancel.
__device__ __forceinline__ float fast_xielu(float z, float a, float b) {
  const float near0 = z * z * fmaf(z, fmaf(z, fmaf(z, 1.f / 120.f, 1.f / 24.f), 1.f / 6.f), 0.5f);
  const float low = z > -0.0625f ? near0 : __expf(z) - 1.f - z;
  return z > 0.f ? fmaf(a * z, z, 0.5f * z) : fmaf(b, low, 0.5f * z);
}

template <typename T, int LANES, int VPL, int ACT>
__global__ void __launch_bounds__(256)
mixer_finish_vec_kernel(const b200_mixer_finish_args a, int norm_blocks) {
  pdl_trigger();
  pdl_wait();
  const int64_t r = blockIdx.y;
  T* o = reinterpret_cast<T*>(a.out) + r * a.out_stride;
  if ((int)blockIdx.x < norm_blocks) {
    __shared__ float red[8];
    const T* y = reinterpret_cast<const T*>(a.y) + r * a.y_stride;
    const T* pre = a.pre_gate ? reinterpret_cast<const T*>(a.pre_gate) + r * a.pre_stride : nullptr;
    const T* post = a.post_gate ? reinterpret_cast<const T*>(a.post_gate) + r * a.post_stride : nullptr;
    const int gs = a.group_size > 0 ? a.group_size : LANES * VPL * 8;
    const int group = blockIdx.x * (256 / LANES) + threadIdx.x / LANES;
    const int c0 = group * gs, c1 = min(c0 + gs, a.inner), first = c0 + (threadIdx.x % LANES) * 8;
    Vec8<T> vy[VPL], vg[VPL];
#pragma unroll
    for (int j = 0; j < VPL; ++j) {
      const int c = first + j * LANES * 8;
      if (c < c1) {
        const int yc = a.y_head_dim > 0 ? c / a.y_head_dim * a.y_head_stride + c % a.y_head_dim : c;
        vy[j] = *reinterpret_cast<const Vec8<T>*>(y + yc);
        if (pre)
          vg[j] = *reinterpret_cast<const Vec8<T>*>(pre + c);
        else if (post)
          vg[j] = *reinterpret_cast<const Vec8<T>*>(post + c);
      }
    }
    float v[VPL][8], ss = 0.f, inv = 1.f;
#pragma unroll
    for (int j = 0; j < VPL; ++j) {
      const bool live = first + j * LANES * 8 < c1;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        v[j][e] = live ? to_float(vy[j].e[e]) : 0.f;
        if (pre && live) {
          const float z = to_float(vg[j].e[e]);
          v[j][e] *= z * fast_sigmoid(z);
        }
        ss += v[j][e] * v[j][e];
      }
    }
    if (a.group_size > 0) {
#pragma unroll
      for (int off = (LANES < 32 ? LANES : 32) / 2; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
      if (LANES > 32) {
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int i = 0; i < (LANES > 32 ? LANES / 32 : 1); ++i) ss += red[threadIdx.x / LANES * (LANES / 32) + i];
      }
      inv = 1.f / sqrtf(ss / (float)gs + a.eps);
    }
#pragma unroll
    for (int j = 0; j < VPL; ++j) {
      const int c = first + j * LANES * 8;
      if (c >= c1) continue;
      float w[8];
      if (a.weight) {
        *reinterpret_cast<float4*>(w) = *reinterpret_cast<const float4*>(a.weight + c);
        *reinterpret_cast<float4*>(w + 4) = *reinterpret_cast<const float4*>(a.weight + c + 4);
      }
      if (post && pre) vg[j] = *reinterpret_cast<const Vec8<T>*>(post + c);
      Vec8<T> res;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        float x = v[j][e] * inv;
        if (a.weight) x *= w[e];
        if (post) {
          const float z = to_float(vg[j].e[e]), g = fast_sigmoid(z);
          x *= a.post_silu ? z * g : g;
        }
        res.e[e] = from_float<T>(x);
      }
      *reinterpret_cast<Vec8<T>*>(o + c) = res;
    }
  } else {
    const T* in = reinterpret_cast<const T*>(a.act_in) + r * a.act_stride;
    const T* mul = a.act_mul ? reinterpret_cast<const T*>(a.act_mul) + r * a.mul_stride : nullptr;
    const int base = ((int)blockIdx.x - norm_blocks) * ACT * 2048 + threadIdx.x * 8;
    Vec8<T> x[ACT], m[ACT];
#pragma unroll
    for (int j = 0; j < ACT; ++j)
      if (base + j * 2048 < a.act_dim) {
        x[j] = *reinterpret_cast<const Vec8<T>*>(in + base + j * 2048);
        if (mul) m[j] = *reinterpret_cast<const Vec8<T>*>(mul + base + j * 2048);
      }
#pragma unroll
    for (int j = 0; j < ACT; ++j) {
      const int i = base + j * 2048;
      if (i >= a.act_dim) break;
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float z = to_float(x[j].e[e]);
        float v = a.act_kind == kActSilu   ? z * fast_sigmoid(z)
                  : a.act_kind == kActGelu ? gelu_erf_f(z)
                  : a.act_kind == kActTanh ? tanhf(z)
                                           : fast_xielu(z, a.act_a, a.act_b);
        if (mul) v *= to_float(m[j].e[e]);
        x[j].e[e] = from_float<T>(v);
      }
      *reinterpret_cast<Vec8<T>*>(o + a.act_offset + i) = x[j];
    }
  }
  if (blockIdx.x == 0 && a.act_dim > 0)
    for (int c = a.act_offset + a.act_dim + threadIdx.x; c < a.out_cols; c += 256) o[c] = from_float<T>(0.f);
}

template <typename T>
bool finish_vec_ok(const b200_mixer_finish_args& a) {
  auto ok = [](const void* p, int64_t stride) { return !p || (((uintptr_t)p & 15) == 0 && stride % 8 == 0); };
  const int gs = a.group_size > 0 ? a.group_size : 2048;
  return sizeof(T) == 2 && ok(a.y, a.y_stride) && ok(a.pre_gate, a.pre_stride) && ok(a.post_gate, a.post_stride) &&
         ok(a.act_in, a.act_stride) && ok(a.act_mul, a.mul_stride) && ok(a.out, a.out_stride) && ((uintptr_t)a.weight & 15) == 0 && a.inner % 8 == 0 &&
         gs % 8 == 0 && gs <= 8192 && a.act_dim % 8 == 0 && a.act_offset % 8 == 0 && a.y_head_dim % 8 == 0 &&
         a.y_head_stride % 8 == 0 && (a.act_dim > 0 ? a.act_offset : a.out_cols) == a.inner;
}

template <typename T>
int launch_finish_vec(const b200_mixer_finish_args& a, cudaStream_t st) {
  const int gs = a.group_size > 0 ? a.group_size : 2048, groups = a.y ? (a.inner + gs - 1) / gs : 0;
  const int lanes = gs <= 64 ? 8 : gs <= 128 ? 16 : gs <= 256 ? 32 : gs <= 512 ? 64 : gs <= 1024 ? 128 : 256;
  const int vpl = gs <= 2048 ? 1 : gs <= 4096 ? 2 : 4, act = a.rows >= 256 ? 2 : 1;
  const int nb = (groups * lanes + 255) / 256, ab = (a.act_dim + act * 2048 - 1) / (act * 2048);
  auto pick = [&](auto act_tag) {
    constexpr int A = decltype(act_tag)::value;
    return vpl == 4      ? mixer_finish_vec_kernel<T, 256, 4, A>
           : vpl == 2    ? mixer_finish_vec_kernel<T, 256, 2, A>
           : lanes == 8 ? mixer_finish_vec_kernel<T, 8, 1, A>
           : lanes == 16 ? mixer_finish_vec_kernel<T, 16, 1, A>
           : lanes == 32 ? mixer_finish_vec_kernel<T, 32, 1, A>
           : lanes == 64 ? mixer_finish_vec_kernel<T, 64, 1, A>
           : lanes == 128 ? mixer_finish_vec_kernel<T, 128, 1, A>
                          : mixer_finish_vec_kernel<T, 256, 1, A>;
  };
  auto* kern = act == 2 ? pick(std::integral_constant<int, 2>()) : pick(std::integral_constant<int, 1>());
  B200_CUDA_OK(launch_pdl(kern, dim3(nb + ab > 0 ? nb + ab : 1, a.rows), dim3(256), 0, st, a, nb));
  return check_launch("mixer_finish");
}

// ---- causal depthwise convolution -----------------------------------------------------------
// One thread per channel walks kConvTile rows with the taps in registers.  Only the first tile of a segment touches
// the carried inputs, and it takes the new ones straight from the input rows, so the tiles never race.
constexpr int kConvTile = 8;
constexpr int kConvMaxTaps = 16;

template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
causal_conv_kernel(const T* __restrict__ in, const float* __restrict__ weight, const float* __restrict__ bias,
                   T* __restrict__ state, const int32_t* __restrict__ cu, const int32_t* __restrict__ seq_lens,
                   const int32_t* __restrict__ slots, T* __restrict__ out, int channels, int taps_rt,
                   int64_t in_stride, int64_t out_stride, int activation) {
  pdl_trigger();
  pdl_wait();
  const int taps = TAPS > 0 ? TAPS : taps_rt;
  constexpr int CAP = TAPS > 0 ? TAPS : kConvMaxTaps;
  const int s = blockIdx.y;
  const int row0 = cu[s], len = cu[s + 1] - row0;
  const int t0 = blockIdx.z * kConvTile;
  const int c = blockIdx.x * 128 + threadIdx.x;
  if (t0 >= len || c >= channels) return;
  const bool fresh = seq_lens[s] == len;
  T* st = state + (int64_t)slots[s] * (taps - 1) * channels + c;
  const T* x = in + (int64_t)row0 * in_stride + c;
  float w[CAP], win[CAP];
#pragma unroll
  for (int k = 0; k < CAP; ++k) {
    w[k] = k < taps ? weight[(int64_t)k * channels + c] : 0.f;
    win[k] = 0.f;
  }
  // win[k] = input of position t0 - (taps - 1) + k, k < taps - 1
#pragma unroll
  for (int k = 0; k < CAP; ++k) {
    if (k >= taps - 1) break;
    const int t = t0 - (taps - 1) + k;
    if (t >= 0)
      win[k] = to_float(x[(int64_t)t * in_stride]);
    else if (!fresh)
      win[k] = to_float(st[(int64_t)(taps - 1 + t) * channels]);
  }
  if (t0 == 0 && taps > 1) {
    T nv[CAP];
#pragma unroll
    for (int k = 0; k < CAP; ++k) {
      if (k >= taps - 1) break;
      const int t = len - (taps - 1) + k;
      if (t >= 0)
        nv[k] = x[(int64_t)t * in_stride];
      else
        nv[k] = fresh ? from_float<T>(0.f) : st[(int64_t)(taps - 1 + t) * channels];
    }
#pragma unroll
    for (int k = 0; k < CAP; ++k) {
      if (k >= taps - 1) break;
      st[(int64_t)k * channels] = nv[k];
    }
  }
  const float b = bias ? bias[c] : 0.f;
  const int t1 = min(t0 + kConvTile, len);
  for (int t = t0; t < t1; ++t) {
    const float cur = to_float(x[(int64_t)t * in_stride]);
    float acc = b;
#pragma unroll
    for (int k = 0; k < CAP; ++k) {
      if (k >= taps) break;
      acc += w[k] * (k == taps - 1 ? cur : win[k]);
    }
    if (activation) acc *= sigmoid_f(acc);
    out[(int64_t)(row0 + t) * out_stride + c] = from_float<T>(acc);
#pragma unroll
    for (int k = 0; k + 1 < CAP; ++k) {
      if (k >= taps - 1) break;
      win[k] = k == taps - 2 ? cur : win[k + 1];
    }
  }
}

// 16-bit types with whole 16-byte units: 8 channels a thread.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128)
causal_conv_vec_kernel(const T* __restrict__ in, const float* __restrict__ weight, const float* __restrict__ bias,
                       T* __restrict__ state, const int32_t* __restrict__ cu, const int32_t* __restrict__ seq_lens,
                       const int32_t* __restrict__ slots, T* __restrict__ out, int channels, int64_t in_stride,
                       int64_t out_stride, int activation) {
  pdl_trigger();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  float w[TAPS][8], b[8];
  if (c < channels) {  // the weights do not depend on earlier kernels
#pragma unroll
    for (int k = 0; k < TAPS; ++k) {
      *reinterpret_cast<float4*>(w[k]) = *reinterpret_cast<const float4*>(weight + (int64_t)k * channels + c);
      *reinterpret_cast<float4*>(w[k] + 4) = *reinterpret_cast<const float4*>(weight + (int64_t)k * channels + c + 4);
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) b[e] = bias ? bias[c + e] : 0.f;
  }
  pdl_wait();
  const int s = blockIdx.y;
  const int row0 = cu[s], len = cu[s + 1] - row0;
  const int t0 = blockIdx.z * kConvTile;
  if (t0 >= len || c >= channels) return;
  const bool fresh = seq_lens[s] == len;
  T* st = state + (int64_t)slots[s] * (TAPS - 1) * channels + c;
  const T* x = in + (int64_t)row0 * in_stride + c;
  auto zero = [] {
    Vec8<T> z;
#pragma unroll
    for (int e = 0; e < 8; ++e) z.e[e] = from_float<T>(0.f);
    return z;
  };
  auto at = [&](int t) {  // input of position t of the segment, carried or new
    if (t >= 0) return *reinterpret_cast<const Vec8<T>*>(x + (int64_t)t * in_stride);
    return fresh ? zero() : *reinterpret_cast<const Vec8<T>*>(st + (int64_t)(TAPS - 1 + t) * channels);
  };
  Vec8<T> win[TAPS > 1 ? TAPS - 1 : 1];
#pragma unroll
  for (int k = 0; k < TAPS - 1; ++k) win[k] = at(t0 - (TAPS - 1) + k);
  if (t0 == 0 && TAPS > 1) {
    Vec8<T> nv[TAPS > 1 ? TAPS - 1 : 1];
#pragma unroll
    for (int k = 0; k < TAPS - 1; ++k) nv[k] = at(len - (TAPS - 1) + k);
#pragma unroll
    for (int k = 0; k < TAPS - 1; ++k) *reinterpret_cast<Vec8<T>*>(st + (int64_t)k * channels) = nv[k];
  }
  const int n = min(kConvTile, len - t0);
  Vec8<T> rows[kConvTile];
#pragma unroll
  for (int i = 0; i < kConvTile; ++i)
    if (i < n) rows[i] = *reinterpret_cast<const Vec8<T>*>(x + (int64_t)(t0 + i) * in_stride);
#pragma unroll
  for (int i = 0; i < kConvTile; ++i) {
    if (i >= n) break;
    const int t = t0 + i;
    const Vec8<T> cur = rows[i];
    Vec8<T> res;
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      float acc = b[e];
#pragma unroll
      for (int k = 0; k < TAPS - 1; ++k) acc += w[k][e] * to_float(win[k].e[e]);
      acc += w[TAPS - 1][e] * to_float(cur.e[e]);
      if (activation) acc *= fast_sigmoid(acc);
      res.e[e] = from_float<T>(acc);
    }
    *reinterpret_cast<Vec8<T>*>(out + (int64_t)(row0 + t) * out_stride + c) = res;
#pragma unroll
    for (int k = 0; k < TAPS - 1; ++k) {
      if (k == TAPS - 2)
        win[k] = cur;
      else
        win[k] = win[k + 1];
    }
  }
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_embed_rows(const int32_t* ids, const void* table, float* out, int rows, int vocab, int dim,
                    int64_t out_stride, int dtype, void* stream) {
  B200_CHECK_ARG(ids && table && out && vocab > 0 && dim > 0, "embed_rows: bad arguments");
  if (rows <= 0) return B200_OK;
  return B200_DISPATCH_DTYPE(dtype, T, [&]() -> int {
    B200_CUDA_OK(launch_pdl(embed_rows_kernel<T>, dim3(rows), dim3(256), 0, (cudaStream_t)stream, ids,
                            (const T*)table, out, vocab, dim, out_stride));
    return check_launch("embed_rows");
  });
}

int b200_stream_norm(const float* x, const int64_t* row_ids, const float* weight, void* out, int rows, int dim,
                     int64_t x_stride, int64_t out_stride, float eps, float weight_offset, int out_dtype,
                     void* stream) {
  B200_CHECK_ARG(x && weight && out && dim > 0, "stream_norm: bad arguments");
  if (rows <= 0) return B200_OK;
  return B200_DISPATCH_DTYPE(out_dtype, T, [&]() -> int {
    const bool vec = dim % 4 == 0 && x_stride % 4 == 0 && out_stride % 4 == 0 &&
                     (((uintptr_t)x | (uintptr_t)weight | (uintptr_t)out) & 15) == 0;
    B200_CUDA_OK(launch_pdl(vec ? stream_norm_kernel<T, true> : stream_norm_kernel<T, false>, dim3(rows), dim3(256),
                            0, (cudaStream_t)stream, x, row_ids, weight, (T*)out, dim, x_stride, out_stride, eps,
                            weight_offset));
    return check_launch("stream_norm");
  });
}

int b200_mixer_finish(const b200_mixer_finish_args* a, void* stream) {
  B200_CHECK_ARG(a && a->out, "mixer_finish: no output");
  B200_CHECK_ARG(a->act_dim == 0 || a->act_in, "mixer_finish: no activation input");
  B200_CHECK_ARG(a->act_kind >= kActGelu && a->act_kind <= kActXielu, "mixer_finish: unknown activation %d", a->act_kind);
  B200_CHECK_ARG(a->group_size >= 0 && (a->group_size == 0 || a->inner % a->group_size == 0),
                 "mixer_finish: inner %d is not a multiple of the group size %d", a->inner, a->group_size);
  B200_CHECK_ARG(a->out_cols >= a->inner && (a->act_dim == 0 || (a->act_offset >= a->inner &&
                                                                  a->out_cols >= a->act_offset + a->act_dim)),
                 "mixer_finish: overlapping or short output columns");
  if (a->rows <= 0 || a->out_cols <= 0) return B200_OK;
  B200_CHECK_ARG(a->rows <= 65535, "mixer_finish: more than 65535 rows");
  const int gs = a->group_size > 0 ? a->group_size : 256;
  const int groups = a->y ? (a->inner + gs - 1) / gs : 0;
  const bool warp = gs <= 512;
  const int nb = warp ? (groups + 7) / 8 : groups;
  const int ab = (a->act_dim + 1023) / 1024;
  const int grid = nb + ab > 0 ? nb + ab : 1;
  return B200_DISPATCH_DTYPE(a->dtype, T, [&]() -> int {
    if (finish_vec_ok<T>(*a)) return launch_finish_vec<T>(*a, (cudaStream_t)stream);
    B200_CUDA_OK(launch_pdl(warp ? mixer_finish_kernel<T, true> : mixer_finish_kernel<T, false>,
                            dim3(grid, a->rows), dim3(256), 0, (cudaStream_t)stream, *a, nb));
    return check_launch("mixer_finish");
  });
}

int b200_causal_conv(const void* in, const float* weight, const float* bias, void* state, const int32_t* cu_seqlens,
                     const int32_t* seq_lens, const int32_t* slots, void* out, int num_seqs, int max_q_len,
                     int channels, int taps, int64_t in_stride, int64_t out_stride, int activation, int dtype,
                     void* stream) {
  B200_CHECK_ARG(in && weight && out && cu_seqlens && seq_lens && slots && channels > 0, "causal_conv: bad arguments");
  B200_CHECK_ARG(taps >= 1 && taps <= kConvMaxTaps, "causal_conv: taps %d outside 1..%d", taps, kConvMaxTaps);
  B200_CHECK_ARG(taps == 1 || state, "causal_conv: no state");
  if (num_seqs <= 0 || max_q_len <= 0) return B200_OK;
  B200_CHECK_ARG(num_seqs <= 65535 && (max_q_len + kConvTile - 1) / kConvTile <= 65535, "causal_conv: batch too large");
  const dim3 grid((channels + 127) / 128, num_seqs, (max_q_len + kConvTile - 1) / kConvTile);
  return B200_DISPATCH_DTYPE(dtype, T, [&]() -> int {
    if (sizeof(T) == 2 && taps >= 2 && taps <= 4 && channels % 8 == 0 && in_stride % 8 == 0 && out_stride % 8 == 0 &&
        (((uintptr_t)in | (uintptr_t)out | (uintptr_t)state | (uintptr_t)weight) & 15) == 0) {
      auto* kern = taps == 4   ? causal_conv_vec_kernel<T, 4>
                   : taps == 3 ? causal_conv_vec_kernel<T, 3>
                               : causal_conv_vec_kernel<T, 2>;
      B200_CUDA_OK(launch_pdl(kern, dim3((channels + 1023) / 1024, grid.y, grid.z), dim3(128), 0, (cudaStream_t)stream,
                              (const T*)in, weight, bias, (T*)state, cu_seqlens, seq_lens, slots, (T*)out, channels,
                              in_stride, out_stride, activation));
      return check_launch("causal_conv");
    }
    auto* kern = taps == 4   ? causal_conv_kernel<T, 4>
                 : taps == 3 ? causal_conv_kernel<T, 3>
                 : taps == 2 ? causal_conv_kernel<T, 2>
                             : causal_conv_kernel<T, 0>;
    B200_CUDA_OK(launch_pdl(kern, grid, dim3(128), 0, (cudaStream_t)stream, (const T*)in, weight, bias, (T*)state,
                            cu_seqlens, seq_lens, slots, (T*)out, channels, taps, in_stride, out_stride, activation));
    return check_launch("causal_conv");
  });
}

}  // extern "C"
