// Shared by the sequential and the chunked form of the gated linear recurrence.
#pragma once

#include "../../include/b200_hybrid_ops.h"
#include "common.cuh"

namespace b200 {
namespace rec {

constexpr int kSsd = 0;
constexpr int kMlstm = 1;
constexpr int kLightning = 2;  // decay per head, no gates
constexpr int kWkv = 3;        // decay per head, key channel and row; a bonus for the current row
constexpr int kTileV = 64;  // value columns per CTA; mLSTM's normaliser state has one copy per tile

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }

template <int VEC>
__device__ __forceinline__ void load_vec(float* d, const float* p) {
  if (VEC == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    d[0] = v.x, d[1] = v.y, d[2] = v.z, d[3] = v.w;
  } else {
    d[0] = *p;
  }
}
template <int VEC>
__device__ __forceinline__ void store_vec(float* p, const float* d) {
  if (VEC == 4)
    *reinterpret_cast<float4*>(p) = make_float4(d[0], d[1], d[2], d[3]);
  else
    *p = d[0];
}

}  // namespace rec
}  // namespace b200
