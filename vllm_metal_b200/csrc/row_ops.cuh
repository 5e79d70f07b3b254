// Helpers of the kernels that work on whole rows: sums over the CTA, 4-column units of fp32 and 16-bit types.
#pragma once

#include "common.cuh"

namespace b200 {
namespace {

// Sums of K values over the CTA, all threads get them; `red` holds K * THREADS / 32 floats and is free again on return.
template <int THREADS, int K>
__device__ __forceinline__ void block_sums(float (&v)[K], float* red) {
  constexpr int W = THREADS / 32;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
  for (int k = 0; k < K; ++k) v[k] = warp_sum(v[k]);
  if (lane == 0)
#pragma unroll
    for (int k = 0; k < K; ++k) red[k * W + warp] = v[k];
  __syncthreads();
#pragma unroll
  for (int k = 0; k < K; ++k) v[k] = warp_sum(lane < W ? red[k * W + lane] : 0.f);
  __syncthreads();
}

__device__ __forceinline__ float gate_f(float z) { return 1.f / (1.f + expf(-z)); }

template <typename T>
__device__ __forceinline__ float4 load4(const T* p) {
  if (sizeof(T) == 4) return *reinterpret_cast<const float4*>(p);
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const T* e = reinterpret_cast<const T*>(&raw);
  return make_float4(to_float(e[0]), to_float(e[1]), to_float(e[2]), to_float(e[3]));
}
template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v) {
  if (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = v;
  } else {
    uint2 raw;
    T* e = reinterpret_cast<T*>(&raw);
    e[0] = from_float<T>(v.x), e[1] = from_float<T>(v.y), e[2] = from_float<T>(v.z), e[3] = from_float<T>(v.w);
    *reinterpret_cast<uint2*>(p) = raw;
  }
}
__device__ __forceinline__ float4 ld4f(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 fma4(float a, float4 x, float4 y) {
  return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w));
}
__device__ __forceinline__ float dot4(float4 x) { return x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w; }

}  // namespace
}  // namespace b200
