// The steps around latent attention (include/b200_hybrid_ops.h): latent norm + rotation + cache write, the per-head
// products into and out of the latent space, and the page gather in front of key / value expansion.
#include "../../include/b200_hybrid_ops.h"
#include "mma_sync.cuh"

namespace b200 {
namespace {

using bf16 = __nv_bfloat16;

// One CTA per row.
template <typename T>
__global__ void __launch_bounds__(128)
latent_prep_kernel(const b200_latent_prep_args a) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[4];
  extern __shared__ float cs[];  // cos, sin of the row's angles
  const int64_t t = blockIdx.x;
  const int half = a.rot_dims >> 1, tid = threadIdx.x;
  const float pos = (float)a.positions[t];
  for (int i = tid; i < half; i += 128) sincosf(pos * a.inv_freq[i], &cs[half + i], &cs[i]);
  const T* down = reinterpret_cast<const T*>(a.down) + t * a.down_stride;
  float ss = 0.f;
  for (int d = tid; d < a.kv_rank; d += 128) {
    const float v = to_float(down[d]);
    ss += v * v;
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  // element d of a rotated vector whose unrotated values come from `src`
  auto rotated = [&](const T* src, int d) {
    if (d >= a.rot_dims) return to_float(src[d]);
    const int i = d >> 1;
    const float u = to_float(src[2 * i]), v = to_float(src[2 * i + 1]), c = cs[i], s = cs[half + i];
    return (d & 1) ? v * c + u * s : u * c - v * s;
  };
  const int64_t slot = a.slot_mapping[t];
  if (slot >= 0 && slot < a.num_slots) {
    T* row = reinterpret_cast<T*>(a.cache) + slot * (a.kv_rank + a.rot_dim);
    const float inv = 1.f / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)a.kv_rank + a.eps);
    for (int d = tid; d < a.kv_rank; d += 128) row[d] = from_float<T>(to_float(down[d]) * inv * a.norm_weight[d]);
    for (int d = tid; d < a.rot_dim; d += 128) row[a.kv_rank + d] = from_float<T>(rotated(down + a.kv_rank, d));
  }
  const T* q = reinterpret_cast<const T*>(a.q) + t * a.q_stride;
  T* o = reinterpret_cast<T*>(a.q_out) + t * a.q_out_stride;
  const int first = a.copy_nope ? 0 : a.rot_offset, span = a.q_cols - first, dh = a.dim + a.rot_dim;
  for (int i = tid; i < a.heads * span; i += 128) {
    const int h = i / span, c = first + i % span;
    const T* qh = q + h * dh;
    float v = 0.f;
    if (c < a.rot_offset)
      v = c < a.dim ? to_float(qh[c]) : 0.f;
    else if (c < a.rot_offset + a.rot_dim)
      v = rotated(qh + a.dim, c - a.rot_offset);
    o[(int64_t)h * a.q_cols + c] = from_float<T>(v);
  }
}

// 16-bit types with whole 16-byte units everywhere: 8 columns a thread and step, whole rotation pairs.
template <typename T>
struct alignas(16) Vec8 {
  T e[8];
};
template <typename T>
__global__ void __launch_bounds__(256)
latent_prep_vec_kernel(const b200_latent_prep_args a) {
  pdl_trigger();
  pdl_wait();
  __shared__ float red[8];
  extern __shared__ float cs[];
  const int64_t t = blockIdx.x;
  const int half = a.rot_dims >> 1, tid = threadIdx.x;
  const float pos = (float)a.positions[t];
  for (int i = tid; i < half; i += 256) sincosf(pos * a.inv_freq[i], &cs[half + i], &cs[i]);
  const T* down = reinterpret_cast<const T*>(a.down) + t * a.down_stride;
  const int64_t slot = a.slot_mapping[t];
  const bool cached = slot >= 0 && slot < a.num_slots;
  Vec8<T> c;
  float ss = 0.f;
  if (tid * 8 < a.kv_rank) {  // kv_rank <= 2048
    c = *reinterpret_cast<const Vec8<T>*>(down + tid * 8);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += to_float(c.e[e]) * to_float(c.e[e]);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  auto rotate = [&](Vec8<T> x, int d) {  // columns d .. d + 7 of the rotated part
#pragma unroll
    for (int e = 0; e < 8; e += 2) {
      if (d + e >= a.rot_dims) break;
      const int i = (d + e) >> 1;
      const float u = to_float(x.e[e]), v = to_float(x.e[e + 1]), co = cs[i], si = cs[half + i];
      x.e[e] = from_float<T>(u * co - v * si);
      x.e[e + 1] = from_float<T>(v * co + u * si);
    }
    return x;
  };
  if (cached) {
    T* row = reinterpret_cast<T*>(a.cache) + slot * (a.kv_rank + a.rot_dim);
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) total += red[i];
    const float inv = 1.f / sqrtf(total / (float)a.kv_rank + a.eps);
    if (tid * 8 < a.kv_rank) {
#pragma unroll
      for (int e = 0; e < 8; ++e) c.e[e] = from_float<T>(to_float(c.e[e]) * inv * a.norm_weight[tid * 8 + e]);
      *reinterpret_cast<Vec8<T>*>(row + tid * 8) = c;
    }
    for (int d = tid * 8; d < a.rot_dim; d += 2048)
      *reinterpret_cast<Vec8<T>*>(row + a.kv_rank + d) =
          rotate(*reinterpret_cast<const Vec8<T>*>(down + a.kv_rank + d), d);
  }
  const T* q = reinterpret_cast<const T*>(a.q) + t * a.q_stride;
  T* o = reinterpret_cast<T*>(a.q_out) + t * a.q_out_stride;
  const int first = (a.copy_nope ? 0 : a.rot_offset) >> 3, span = (a.q_cols >> 3) - first, dh = a.dim + a.rot_dim;
  for (int i = tid; i < a.heads * span; i += 256) {
    const int h = i / span, col = (first + i - h * span) * 8;
    const T* qh = q + h * dh;
    Vec8<T> v;
#pragma unroll
    for (int e = 0; e < 8; ++e) v.e[e] = from_float<T>(0.f);
    if (col < a.rot_offset) {
      if (col < a.dim) v = *reinterpret_cast<const Vec8<T>*>(qh + col);
    } else if (col < a.rot_offset + a.rot_dim) {
      v = rotate(*reinterpret_cast<const Vec8<T>*>(qh + a.dim + col - a.rot_offset), col - a.rot_offset);
    }
    *reinterpret_cast<Vec8<T>*>(o + (int64_t)h * a.q_cols + col) = v;
  }
}

__device__ __forceinline__ float gate_value(const void* gate, int64_t off, int is_f32, int is_half) {
  const float z = is_f32    ? reinterpret_cast<const float*>(gate)[off]
                  : is_half ? to_float(reinterpret_cast<const __half*>(gate)[off])
                            : to_float(reinterpret_cast<const bf16*>(gate)[off]);
  return 1.f / (1.f + expf(-z));
}

// Any type and size: one warp per output, lanes over k.
template <typename T>
__global__ void __launch_bounds__(256)
head_linear_kernel(const b200_head_linear_args a) {
  pdl_trigger();
  pdl_wait();
  const int64_t t = blockIdx.z;
  const int h = blockIdx.y, n = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (n >= a.n) return;
  const T* x = reinterpret_cast<const T*>(a.x) + t * a.x_stride + h * a.x_head_stride;
  const T* w = reinterpret_cast<const T*>(a.w) + ((int64_t)h * a.n + n) * a.k;
  float acc = 0.f;
  for (int k = lane; k < a.k; k += 32) acc += to_float(w[k]) * to_float(x[k]);
  acc = warp_sum(acc);
  if (lane == 0) {
    if (a.gate)
      acc *= gate_value(a.gate, t * a.gate_stride + (int64_t)h * a.n + n, TypeTag<T>::value == B200_F32,
                        TypeTag<T>::value == B200_F16);
    reinterpret_cast<T*>(a.y)[t * a.y_stride + h * a.y_head_stride + n] = from_float<T>(acc);
  }
}

// bf16 on tensor cores: 64 rows x 32 outputs of one head per CTA, 64-wide k slabs in a ring of four.
constexpr int kPad = 72, kCols = 32, kRing = 4;
constexpr int kHeadLinearSmem = kRing * (64 + kCols) * kPad * 2;
__global__ void __launch_bounds__(128)
head_linear_mma_kernel(const b200_head_linear_args a, int pairs) {
  extern __shared__ __align__(16) uint8_t hl_raw[];
  bf16* sx = reinterpret_cast<bf16*>(hl_raw);
  bf16* sw = sx + kRing * 64 * kPad;
  pdl_trigger();
  const int h = blockIdx.y, n0 = blockIdx.x * kCols, r0 = blockIdx.z * 64;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bf16* x = reinterpret_cast<const bf16*>(a.x) + (int64_t)r0 * a.x_stride + h * a.x_head_stride;
  const bf16* w = reinterpret_cast<const bf16*>(a.w) + ((int64_t)h * a.n + n0) * a.k;
  const int rows = min(64, a.rows - r0), cols = min(kCols, a.n - n0), slabs = (a.k + 63) / 64;
  auto load_w = [&](int s) {
    for (int i = tid; i < kCols * 8; i += 128) {
      const int r = i >> 3, c = (i & 7) * 8;
      const bool live = r < cols && s * 64 + c < a.k;
      mma::cp_async16(&sw[((s % kRing) * kCols + r) * kPad + c], live ? w + (int64_t)r * a.k + s * 64 + c : w, live);
    }
  };
  auto load_x = [&](int s) {
    for (int i = tid; i < 512; i += 128) {
      const int r = i >> 3, c = (i & 7) * 8;
      const bool live = r < rows && s * 64 + c < a.k;
      mma::cp_async16(&sx[((s % kRing) * 64 + r) * kPad + c], live ? x + (int64_t)r * a.x_stride + s * 64 + c : x, live);
    }
  };
  for (int s = 0; s < kRing - 1 && s < slabs; ++s) load_w(s);  // weights do not depend on the previous kernel
  pdl_wait();
  for (int s = 0; s < kRing - 1; ++s) {
    if (s < slabs) load_x(s);
    mma::cp_commit();  // the weights ride in the first group: waiting for it means waiting for all of them
  }
  float acc[4][4];
#pragma unroll
  for (int n = 0; n < 4; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
  for (int s = 0; s < slabs; ++s) {
    mma::cp_wait<kRing - 2>();
    __syncthreads();
    if (s + kRing - 1 < slabs) {
      load_w(s + kRing - 1);
      load_x(s + kRing - 1);
    }
    mma::cp_commit();
    const bf16 *xs = sx + (s % kRing) * 64 * kPad, *wsm = sw + (s % kRing) * kCols * kPad;
#pragma unroll
    for (int ks = 0; ks < 4; ++ks) {
      uint32_t fa[4];
      mma::ldsm4(fa, &xs[(warp * 16 + (lane & 15)) * kPad + ks * 16 + (lane >> 4) * 8]);
#pragma unroll
      for (int n2 = 0; n2 < 2; ++n2) {
        uint32_t fb[4];
        mma::ldsm4(fb, &wsm[(n2 * 16 + (lane >> 4) * 8 + (lane & 7)) * kPad + ks * 16 + ((lane >> 3) & 1) * 8]);
        mma::mma16816(acc[2 * n2], fa, fb[0], fb[1]);
        mma::mma16816(acc[2 * n2 + 1], fa, fb[2], fb[3]);
      }
    }
  }
#pragma unroll
  for (int n = 0; n < 4; ++n)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = warp * 16 + (lane >> 2) + e * 8, c = n0 + n * 8 + (lane & 3) * 2;
      if (r >= rows || c >= a.n) continue;
      const int64_t t = r0 + r, off = t * a.gate_stride + (int64_t)h * a.n + c;
      float u = acc[n][2 * e], v = acc[n][2 * e + 1];
      bf16* y = reinterpret_cast<bf16*>(a.y) + t * a.y_stride + h * a.y_head_stride + c;
      if (pairs) {  // whole aligned pairs
        if (a.gate) {
          const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(reinterpret_cast<const bf16*>(a.gate) + off));
          u *= 1.f / (1.f + expf(-z.x));
          v *= 1.f / (1.f + expf(-z.y));
        }
        *reinterpret_cast<__nv_bfloat162*>(y) = __floats2bfloat162_rn(u, v);
      } else {
        if (a.gate) u *= gate_value(a.gate, off, 0, 0);
        y[0] = __float2bfloat16_rn(u);
        if (c + 1 < a.n) {
          if (a.gate) v *= gate_value(a.gate, off + 1, 0, 0);
          y[1] = __float2bfloat16_rn(v);
        }
      }
    }
}

// One warp per gathered row (blockIdx.x * 8 + warp), request blockIdx.y.
template <typename T>
__global__ void __launch_bounds__(256)
latent_gather_kernel(const T* __restrict__ cache, const int32_t* __restrict__ tables, const int32_t* __restrict__ first,
                     const int32_t* __restrict__ count, const int32_t* __restrict__ out_row, T* __restrict__ out,
                     int width, int block_size, int max_blocks, int64_t num_slots, int pad) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.y, i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  const int n = count[s], padded = (n + pad - 1) / pad * pad;
  if (i >= padded) return;
  T* o = out + (int64_t)(out_row[s] + i) * width;
  const int j = first[s] + i;
  const int64_t slot = i < n ? (int64_t)tables[(int64_t)s * max_blocks + j / block_size] * block_size + j % block_size : -1;
  const bool live = slot >= 0 && slot < num_slots;
  const T* src = cache + (live ? slot : 0) * width;
  constexpr int VE = 16 / (int)sizeof(T);
  if (width % VE == 0) {
    for (int c = lane; c < width / VE; c += 32)
      reinterpret_cast<uint4*>(o)[c] = live ? reinterpret_cast<const uint4*>(src)[c] : make_uint4(0, 0, 0, 0);
  } else {
    for (int c = lane; c < width; c += 32) o[c] = live ? src[c] : from_float<T>(0.f);
  }
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_latent_prep(const b200_latent_prep_args* a, void* stream) {
  B200_CHECK_ARG(a && a->q && a->down && a->positions && a->cache && a->slot_mapping && a->norm_weight && a->q_out,
                 "latent_prep: null argument");
  B200_CHECK_ARG(a->rot_dims >= 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->rot_dim, "latent_prep: rot_dims %d of %d",
                 a->rot_dims, a->rot_dim);
  B200_CHECK_ARG(a->rot_dims == 0 || a->inv_freq, "latent_prep: no frequencies");
  B200_CHECK_ARG(a->q_cols >= a->rot_offset + a->rot_dim && (!a->copy_nope || a->rot_offset >= a->dim),
                 "latent_prep: query columns overlap");
  if (a->num_tokens <= 0) return B200_OK;
  auto ok = [](const void* p, int64_t stride) { return ((uintptr_t)p & 15) == 0 && stride % 8 == 0; };
  const bool vec = ok(a->q, a->q_stride) && ok(a->down, a->down_stride) && ok(a->cache, 0) && ok(a->q_out, a->q_out_stride) &&
                   a->dim % 8 == 0 && a->rot_dim % 8 == 0 && a->kv_rank % 8 == 0 && a->kv_rank <= 2048 &&
                   a->q_cols % 8 == 0 && a->rot_offset % 8 == 0;
  return B200_DISPATCH_DTYPE(a->dtype, T, [&]() -> int {
    if (vec && sizeof(T) == 2) {
      B200_CUDA_OK(launch_pdl(latent_prep_vec_kernel<T>, dim3(a->num_tokens), dim3(256), a->rot_dims * sizeof(float),
                              (cudaStream_t)stream, *a));
      return check_launch("latent_prep");
    }
    B200_CUDA_OK(launch_pdl(latent_prep_kernel<T>, dim3(a->num_tokens), dim3(128), a->rot_dims * sizeof(float),
                            (cudaStream_t)stream, *a));
    return check_launch("latent_prep");
  });
}

int b200_head_linear(const b200_head_linear_args* a, void* stream) {
  B200_CHECK_ARG(a && a->x && a->w && a->y && a->n > 0 && a->k > 0 && a->heads > 0, "head_linear: bad arguments");
  if (a->rows <= 0) return B200_OK;
  auto ok = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  if (a->dtype == B200_BF16 && a->k % 8 == 0 && a->x_stride % 8 == 0 && a->x_head_stride % 8 == 0 && ok(a->x) && ok(a->w)) {
    const dim3 grid((a->n + kCols - 1) / kCols, a->heads, (a->rows + 63) / 64);
    const int pairs = a->n % 2 == 0 && a->y_stride % 2 == 0 && a->y_head_stride % 2 == 0 && a->gate_stride % 2 == 0 &&
                      (((uintptr_t)a->y | (uintptr_t)a->gate) & 3) == 0;
    static bool attr = false;
    if (!attr) {
      B200_CUDA_OK(cudaFuncSetAttribute(head_linear_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kHeadLinearSmem));
      attr = true;
    }
    B200_CUDA_OK(launch_pdl(head_linear_mma_kernel, grid, dim3(128), kHeadLinearSmem, (cudaStream_t)stream, *a, pairs));
    return check_launch("head_linear (mma)");
  }
  B200_CHECK_ARG(a->rows <= 65535, "head_linear: more than 65535 rows");
  return B200_DISPATCH_DTYPE(a->dtype, T, [&]() -> int {
    B200_CUDA_OK(launch_pdl(head_linear_kernel<T>, dim3((a->n + 7) / 8, a->heads, a->rows), dim3(256), 0,
                            (cudaStream_t)stream, *a));
    return check_launch("head_linear");
  });
}

int b200_latent_gather(const void* cache, const int32_t* block_tables, const int32_t* first, const int32_t* count,
                       const int32_t* out_row, void* out, int num_seqs, int max_count, int width, int block_size,
                       int max_blocks_per_seq, int64_t num_slots, int pad, int dtype, void* stream) {
  B200_CHECK_ARG(cache && block_tables && first && count && out_row && out && width > 0 && block_size > 0 && pad > 0,
                 "latent_gather: bad arguments");
  if (num_seqs <= 0 || max_count <= 0) return B200_OK;
  const int padded = (max_count + pad - 1) / pad * pad;
  return B200_DISPATCH_DTYPE(dtype, T, [&]() -> int {
    B200_CUDA_OK(launch_pdl(latent_gather_kernel<T>, dim3((padded + 7) / 8, num_seqs), dim3(256), 0,
                            (cudaStream_t)stream, (const T*)cache, block_tables, first, count, out_row, (T*)out, width,
                            block_size, max_blocks_per_seq, num_slots, pad));
    return check_launch("latent_gather");
  });
}

}  // extern "C"
