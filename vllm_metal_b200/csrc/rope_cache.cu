// Fused per-head RMSNorm -> RoPE -> KV-cache write.
//
// One launch does what the reference's sdpa_forward does in five steps between the q/k/v
// projections and the attention kernel (vllm_metal/attention/impls/sdpa.py:348-368 q/k norm +
// RoPE, :542-544 cast, :638 reshape_and_cache -> kernels_v2/reshape_and_cache.metal:36-96):
//
//   q[t,h,:]  <- rope(norm(q[t,h,:]))                       in place (strided rows of the qkv buffer)
//   k[t,h,:]  <- rope(norm(k[t,h,:]))                       in place AND to key_cache[slot[t]]
//   value_cache[slot[t]] <- v[t,:,:]                        bit-exact copy
//
// The arithmetic is the composition of the standalone ops bit for bit: the norm result is
// rounded to T before the rotation reads it, angles come from the same fp32 formula as
// rope_kernel, slot < 0 (padding) skips the cache write only.  One CTA per token, one warp per
// head; a head row is staged in shared memory as fp32 so any head_dim / rot_dim / pair layout
// works.  HBM bytes per token: (Hq + 2*Hkv)*D*esize read, (Hq + Hkv)*D*esize in-place write,
// 2*Hkv*D*esize cache write.
#include "common.cuh"
#include "../../include/b200_decoder_ops.h"
#include "../../include/b200_hybrid_ops.h"

namespace b200 {

constexpr int RC_MAX_D = 512;
constexpr int RC_WARPS = 8;

template <typename T>
__global__ void __launch_bounds__(RC_WARPS * 32)
norm_rope_cache_kernel(T* __restrict__ q, T* __restrict__ k, const T* __restrict__ v,
                       const T* __restrict__ q_norm_w, const T* __restrict__ k_norm_w,
                       const int32_t* __restrict__ positions, const int64_t* __restrict__ slot_mapping,
                       T* __restrict__ key_cache, T* __restrict__ value_cache, int num_q_heads,
                       int num_kv_heads, int head_dim, int rot_dim, float log2_base, int traditional,
                       float eps, int64_t q_stride, int64_t k_stride, int64_t v_stride, int block_size,
                       int64_t num_slots, int64_t kv_block_stride, int64_t kv_token_stride, int value_dim,
                       int64_t v_block_stride, int64_t v_token_stride) {
  pdl_trigger();
  pdl_wait();
  __shared__ float rows[RC_WARPS][RC_MAX_D];
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float pos = positions ? (float)positions[t] : 0.f;
  const int64_t slot = slot_mapping ? slot_mapping[t] : -1;
  const bool write_cache = slot >= 0 && slot < num_slots;
  int64_t cache_off = 0, v_off = 0;
  if (write_cache) {
    const int64_t blk = slot / block_size;
    cache_off = blk * kv_block_stride + (slot - blk * block_size) * kv_token_stride;
    v_off = blk * v_block_stride + (slot - blk * block_size) * v_token_stride;
  }
  const int half = rot_dim >> 1;
  float* row = rows[warp];
  const int total = num_q_heads + 2 * num_kv_heads;
  // heads are spread over gridDim.y CTAs per token so a 64-token decode step fills the machine
  for (int h = blockIdx.y * RC_WARPS + warp; h < total; h += RC_WARPS * gridDim.y) {
    if (h >= num_q_heads + num_kv_heads) {
      // ---- V head: bit-exact copy into the cache ----
      if (!write_cache) continue;
      const int hv = h - num_q_heads - num_kv_heads;
      const T* src = v + (int64_t)t * v_stride + (int64_t)hv * value_dim;
      T* dst = value_cache + v_off + (int64_t)hv * value_dim;
      if (sizeof(T) == 2 && value_dim % 8 == 0 && ((uintptr_t)src % 16 == 0) && ((uintptr_t)dst % 16 == 0)) {
        for (int i = lane; i < value_dim / 8; i += 32)
          reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
      } else {
        for (int i = lane; i < value_dim; i += 32) dst[i] = src[i];
      }
      continue;
    }
    const bool is_q = h < num_q_heads;
    T* base = is_q ? q + (int64_t)t * q_stride + (int64_t)h * head_dim
                   : k + (int64_t)t * k_stride + (int64_t)(h - num_q_heads) * head_dim;
    const T* nw = is_q ? q_norm_w : k_norm_w;
    const bool do_norm = is_q ? (q_norm_w != nullptr) : (k_norm_w != nullptr);
    // ---- load (+ per-head RMSNorm, rounded to T like the standalone op) ----
    float ss = 0.f;
    for (int i = lane; i < head_dim; i += 32) {
      const float x = to_float(base[i]);
      row[i] = x;
      ss += x * x;
    }
    if (do_norm) {
      ss = warp_sum(ss);
      const float inv = rsqrtf(ss / (float)head_dim + eps);
      for (int i = lane; i < head_dim; i += 32)
        row[i] = to_float(from_float<T>(row[i] * inv * to_float(nw[i])));
    }
    __syncwarp();
    T* cdst = (!is_q && write_cache) ? key_cache + cache_off + (int64_t)(h - num_q_heads) * head_dim : nullptr;
    // ---- rotate the first rot_dim dims ----
    for (int i = lane; i < half; i += 32) {
      const float inv_freq = exp2f(-log2_base * (2.f * (float)i / (float)rot_dim));
      float sn, cs;
      sincosf(pos * inv_freq, &sn, &cs);
      const int i0 = traditional ? 2 * i : i;
      const int i1 = traditional ? 2 * i + 1 : i + half;
      const float a = row[i0], b = row[i1];
      const T o0 = from_float<T>(a * cs - b * sn), o1 = from_float<T>(b * cs + a * sn);
      base[i0] = o0;
      base[i1] = o1;
      if (cdst) {
        cdst[i0] = o0;
        cdst[i1] = o1;
      }
    }
    // ---- pass-through dims (rot_dim < head_dim, or no RoPE at all) ----
    for (int i = rot_dim + lane; i < head_dim; i += 32) {
      const T o = from_float<T>(row[i]);
      if (do_norm) base[i] = o;
      if (cdst) cdst[i] = o;
    }
    __syncwarp();
  }
}

// ---- the other order: RoPE (if any) -> per-head norm -> cache ------------------------------------------
// Angles from a frequency table (scaled rotations), once per token and CTA.  One CTA per token, a warp per head, a lane
// holds the pairs lane, lane + 32, ... of the head in registers from load to store.
template <typename T>
struct alignas(2 * sizeof(T)) Pair {
  T a, b;
};
template <typename T, int NP, bool VEC>
__device__ __forceinline__ void load_pairs(const T* src, int dim, float2 (&v)[NP]) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int j = 0; j < NP; ++j) {
    const int e = 2 * (lane + 32 * j);
    v[j] = make_float2(0.f, 0.f);
    if (VEC) {
      if (e < dim) {
        const Pair<T> p = *reinterpret_cast<const Pair<T>*>(src + e);
        v[j] = make_float2(to_float(p.a), to_float(p.b));
      }
    } else {
      if (e < dim) v[j].x = to_float(src[e]);
      if (e + 1 < dim) v[j].y = to_float(src[e + 1]);
    }
  }
}

// times `f` and, where given, a weight per dimension
template <typename T, int NP, bool VEC>
__device__ __forceinline__ void store_pairs(T* dst, int dim, const float2 (&v)[NP], float f, const float* weight) {
  const int lane = threadIdx.x & 31;
#pragma unroll
  for (int j = 0; j < NP; ++j) {
    const int e = 2 * (lane + 32 * j);
    if (e >= dim) continue;
    const float x = v[j].x * f * (weight ? weight[e] : 1.f), y = v[j].y * f * (weight && e + 1 < dim ? weight[e + 1] : 1.f);
    if (VEC) {
      *reinterpret_cast<Pair<T>*>(dst + e) = Pair<T>{from_float<T>(x), from_float<T>(y)};
    } else {
      dst[e] = from_float<T>(x);
      if (e + 1 < dim) dst[e + 1] = from_float<T>(y);
    }
  }
}

template <typename T, int NP, bool VEC>
__global__ void __launch_bounds__(RC_WARPS * 32)
rope_norm_cache_kernel(const b200_rope_norm_cache_args a) {
  __shared__ float2 turn[RC_MAX_D / 2];  // factor * (cos, sin)
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float pos = (float)a.positions[t];
  for (int i = threadIdx.x; 2 * i < a.rot_dims; i += RC_WARPS * 32) {
    // what the rounded product and the frequency's low part leave of the angle, r, turns it by a Taylor step
    const float hi = a.freq[2 * i], ang = pos * hi, r = fmaf(pos, a.freq[2 * i + 1], fmaf(pos, hi, -ang));
    float sn, cs;
    sincosf(ang, &sn, &cs);
    const float s1 = fmaf(-r * r, r * (1.f / 6.f), r), c1 = -0.5f * r * r;  // sin r, cos r - 1
    turn[i] = make_float2(a.rot_factor * (cs + fmaf(-s1, sn, c1 * cs)), a.rot_factor * (sn + fmaf(s1, cs, c1 * sn)));
  }
  __syncthreads();
  float temp = 1.f;
  if (a.temp_coef != 0.f) temp = 1.f + a.temp_coef * logf((float)floor(((double)a.positions[t] + 1.0) / (double)a.temp_every) + 1.f);
  const int64_t slot = a.slot_mapping[t];
  const bool cached = slot >= 0 && slot < a.num_blocks * a.block_size;
  const int64_t blk = cached ? slot / a.block_size : 0, off = cached ? slot - blk * a.block_size : 0;
  T* krow = reinterpret_cast<T*>(a.key_cache) + blk * a.k_block_stride + off * a.k_token_stride;
  T* vrow = reinterpret_cast<T*>(a.value_cache) + blk * a.v_block_stride + off * a.v_token_stride;
  for (int h = blockIdx.y * RC_WARPS + warp; h < a.heads + 2 * a.kv_heads; h += RC_WARPS * gridDim.y) {
    if (h >= a.heads + a.kv_heads) {
      const int hv = h - a.heads - a.kv_heads;
      const T* src = reinterpret_cast<const T*>(a.v) + (int64_t)t * a.v_stride + (int64_t)hv * a.vdim;
      T* dst = vrow + (int64_t)hv * a.vdim;
      if (!cached) continue;
      if (a.norm_values) {
        float2 v[NP];
        load_pairs<T, NP, VEC>(src, a.vdim, v);
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < NP; ++j) ss += v[j].x * v[j].x + v[j].y * v[j].y;
        store_pairs<T, NP, VEC>(dst, a.vdim, v, 1.f / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps), nullptr);
        continue;
      }
      if (a.vdim % (16 / sizeof(T)) == 0 && (((uintptr_t)src | (uintptr_t)dst) & 15) == 0) {
        for (int i = lane; i < a.vdim / (int)(16 / sizeof(T)); i += 32)
          reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
      } else {
        for (int i = lane; i < a.vdim; i += 32) dst[i] = src[i];
      }
      continue;
    }
    const bool is_q = h < a.heads;
    if (!is_q && !cached) continue;
    T* qrow = reinterpret_cast<T*>(a.q) + (int64_t)t * a.q_stride + (int64_t)h * a.dim;
    const T* src = is_q ? qrow : reinterpret_cast<const T*>(a.k) + (int64_t)t * a.k_stride + (int64_t)(h - a.heads) * a.dim;
    T* dst = is_q ? qrow : krow + (int64_t)(h - a.heads) * a.dim;
    float2 v[NP];
    load_pairs<T, NP, VEC>(src, a.dim, v);
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NP; ++j) {
      const int i = lane + 32 * j;
      if (2 * i < a.rot_dims) {
        const float2 w = turn[i];
        v[j] = make_float2(v[j].x * w.x - v[j].y * w.y, v[j].y * w.x + v[j].x * w.y);
      }
      ss += v[j].x * v[j].x + v[j].y * v[j].y;
    }
    float f = 1.f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
    if (is_q && a.q_weight) f *= a.q_weight[h];
    if (is_q) f *= temp;
    store_pairs<T, NP, VEC>(dst, a.dim, v, f, is_q ? a.q_norm : a.k_norm);
  }
}

template <typename T, bool VEC>
int launch_rope_norm_cache(const b200_rope_norm_cache_args& a, cudaStream_t st) {
  const int total = a.heads + 2 * a.kv_heads, need = (total + RC_WARPS - 1) / RC_WARPS;
  const dim3 grid(a.num_tokens, a.num_tokens >= 1024 ? 1 : need);
  const int held = a.norm_values && a.vdim > a.dim ? a.vdim : a.dim;
  auto* kern = held <= 64    ? rope_norm_cache_kernel<T, 1, VEC>
               : held <= 128 ? rope_norm_cache_kernel<T, 2, VEC>
               : held <= 256 ? rope_norm_cache_kernel<T, 4, VEC>
                              : rope_norm_cache_kernel<T, 8, VEC>;
  B200_CUDA_OK(launch_pdl(kern, grid, dim3(RC_WARPS * 32), 0, st, a));
  return check_launch("rope_norm_cache");
}

}  // namespace b200

extern "C" int b200_rope_norm_cache(const b200_rope_norm_cache_args* a, void* stream) {
  using namespace b200;
  B200_CHECK_ARG(a && a->q && a->k && a->v && a->key_cache && a->value_cache && a->positions && a->slot_mapping,
                 "rope_norm_cache: null pointer argument");
  B200_CHECK_ARG(a->heads > 0 && a->kv_heads > 0 && a->vdim > 0 && a->dim > 0 && a->dim <= RC_MAX_D,
                 "rope_norm_cache: head size must be in [1, %d], got %d (heads %d/%d)", RC_MAX_D, a->dim, a->heads, a->kv_heads);
  B200_CHECK_ARG(a->rot_dims >= 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->dim && (a->rot_dims == 0 || a->freq),
                 "rope_norm_cache: %d rotated of %d dimensions", a->rot_dims, a->dim);
  B200_CHECK_ARG(a->block_size > 0 && a->num_blocks > 0 && a->k_token_stride >= (int64_t)a->kv_heads * a->dim &&
                     a->v_token_stride >= (int64_t)a->kv_heads * a->vdim,
                 "rope_norm_cache: bad cache geometry");
  B200_CHECK_ARG(!a->norm_values || a->vdim <= RC_MAX_D, "rope_norm_cache: normed values of at most %d columns, got %d", RC_MAX_D,
                 a->vdim);
  B200_CHECK_ARG(a->temp_coef == 0.f || a->temp_every > 0.f, "rope_norm_cache: temp_every must be positive");
  if (a->num_tokens <= 0) return B200_OK;
  return B200_DISPATCH_DTYPE(a->dtype, T, [&]() -> int {
    auto ok = [](const void* p, int64_t s0, int64_t s1) {
      return (uintptr_t)p % (2 * sizeof(T)) == 0 && s0 % 2 == 0 && s1 % 2 == 0;
    };
    const bool vec = a->dim % 2 == 0 && ok(a->q, a->q_stride, 0) && ok(a->k, a->k_stride, 0) &&
                     ok(a->key_cache, a->k_block_stride, a->k_token_stride) &&
                     (!a->norm_values || (a->vdim % 2 == 0 && ok(a->v, a->v_stride, 0) &&
                                          ok(a->value_cache, a->v_block_stride, a->v_token_stride)));
    return vec ? launch_rope_norm_cache<T, true>(*a, (cudaStream_t)stream)
               : launch_rope_norm_cache<T, false>(*a, (cudaStream_t)stream);
  });
}

extern "C" int b200_norm_rope_cache(void* q, void* k, const void* v, const void* q_norm_weight,
                                    const void* k_norm_weight, const int32_t* positions,
                                    const int64_t* slot_mapping, void* key_cache, void* value_cache,
                                    int num_tokens, int num_q_heads, int num_kv_heads, int head_dim,
                                    int rot_dim, float base, int traditional, float eps,
                                    int64_t q_stride, int64_t k_stride, int64_t v_stride,
                                    int block_size, int64_t num_blocks, int64_t kv_block_stride,
                                    int64_t kv_token_stride, int value_dim, int64_t v_block_stride,
                                    int64_t v_token_stride, int dtype, void* stream) {
  using namespace b200;
  B200_CHECK_ARG(num_tokens >= 0, "norm_rope_cache: num_tokens must be >= 0, got %d", num_tokens);
  if (num_tokens == 0) return B200_OK;
  B200_CHECK_ARG(q && k && v && key_cache && value_cache && slot_mapping,
                 "norm_rope_cache: null pointer argument");
  B200_CHECK_ARG(num_q_heads > 0 && num_kv_heads > 0 && head_dim > 0 && head_dim <= RC_MAX_D,
                 "norm_rope_cache: head_dim must be in [1, %d], got %d (heads %d/%d)", RC_MAX_D, head_dim,
                 num_q_heads, num_kv_heads);
  B200_CHECK_ARG(rot_dim >= 0 && rot_dim % 2 == 0 && rot_dim <= head_dim,
                 "norm_rope_cache: rot_dim (%d) must be even and <= head_dim (%d)", rot_dim, head_dim);
  B200_CHECK_ARG(rot_dim == 0 || (positions != nullptr && base > 0.f),
                 "norm_rope_cache: RoPE needs positions and a positive base");
  B200_CHECK_ARG(block_size > 0 && num_blocks > 0, "norm_rope_cache: bad cache geometry");
  const int64_t row_elems = (int64_t)num_kv_heads * head_dim, v_elems = (int64_t)num_kv_heads * value_dim;
  B200_CHECK_ARG(value_dim > 0 && v_token_stride >= v_elems && v_block_stride >= v_token_stride * block_size,
                 "norm_rope_cache: value cache strides overlap (block=%lld token=%lld row=%lld)",
                 (long long)v_block_stride, (long long)v_token_stride, (long long)v_elems);
  B200_CHECK_ARG(kv_token_stride >= row_elems && kv_block_stride >= kv_token_stride * block_size,
                 "norm_rope_cache: cache strides overlap (block=%lld token=%lld row=%lld)",
                 (long long)kv_block_stride, (long long)kv_token_stride, (long long)row_elems);
  cudaStream_t st = (cudaStream_t)stream;
  const float l2b = rot_dim > 0 ? log2f(base) : 0.f;
  return B200_DISPATCH_DTYPE(dtype, T, [&]() -> int {
    const int total_heads = num_q_heads + 2 * num_kv_heads;
    const int ysplit = num_tokens >= 1024 ? 1 : (total_heads + RC_WARPS - 1) / RC_WARPS;
    launch_pdl(norm_rope_cache_kernel<T>, dim3(num_tokens, ysplit), dim3(RC_WARPS * 32), 0, st, 
        (T*)q, (T*)k, (const T*)v, (const T*)q_norm_weight, (const T*)k_norm_weight, positions,
        slot_mapping, (T*)key_cache, (T*)value_cache, num_q_heads, num_kv_heads, head_dim, rot_dim, l2b,
        traditional, eps, q_stride, k_stride, v_stride, block_size, num_blocks * block_size,
        kv_block_stride, kv_token_stride, value_dim, v_block_stride, v_token_stride);
    return check_launch("norm_rope_cache_kernel");
  });
}
