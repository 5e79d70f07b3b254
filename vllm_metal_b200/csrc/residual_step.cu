// The step between two sublayers (include/b200_hybrid_ops.h): the result's norm where the design has one, the sum, the next
// input's norm and, for single rows, the short convolution on that input or its mixes with the row before, in one launch.  A
// result may arrive as the weighted parts of routed experts and a gated shared part.  Token mixes of portions are a kernel of
// their own, below.
//
// PLUS: the forms of pre-norm designs -- results without a norm, a bias, embedding rows and a vector added on the way, norms in
// groups, 32-bit inputs, mixes.  A compile-time form, so that the others stay as they are.
//
// HBM-bound at 2 * dim * 4 bytes a row plus the 16-bit operands; one CTA a row, the row in registers between its norms.
#include "../../include/b200_hybrid_ops.h"
#include "row_ops.cuh"

namespace b200 {
namespace {

constexpr int kMaxStepTaps = 16;

template <typename T>
struct StepRow {  // pointers of one row
  float* x;
  const T *y, *extra;
  const float* pw;
  T *h, *state;
  const T* embed;
  float *h32, *last;
  float gate;
  bool store;
  int seen;  // earlier inputs the sequence has
  __device__ StepRow(const b200_residual_step_args& a) {
    const int64_t b = blockIdx.x, r = a.row_ids ? a.row_ids[b] : b;
    store = !a.row_ids;
    x = a.x + r * a.dim;
    const int64_t first = a.parts > 0 ? r * a.parts : r;
    y = a.y ? reinterpret_cast<const T*>(a.y) + first * a.y_stride : nullptr;
    pw = a.parts > 0 ? a.part_weight + first : nullptr;
    extra = a.extra ? reinterpret_cast<const T*>(a.extra) + r * a.extra_stride : nullptr;
    gate = a.extra ? gate_f(a.extra_gate[r * a.gate_stride]) : 0.f;
    h = a.h ? reinterpret_cast<T*>(a.h) + b * a.h_stride : nullptr;
    state = a.conv_weight && a.taps > 1 ? reinterpret_cast<T*>(a.state) + (int64_t)a.slots[b] * (a.taps - 1) * a.dim : nullptr;
    seen = a.conv_weight || a.mixes > 0 ? a.seq_lens[b] - 1 : 0;
    const int id = a.table ? a.ids[r] : -1;
    embed = id >= 0 && id < a.vocab ? reinterpret_cast<const T*>(a.table) + (int64_t)id * a.dim : nullptr;
    h32 = a.h32 ? a.h32 + b * a.h_stride : nullptr;
    last = a.mixes > 0 ? a.mix_state + (int64_t)a.slots[b] * a.dim : nullptr;
  }
};

template <typename T>
__device__ __forceinline__ float4 round4(float4 v) {
  return make_float4(to_float(from_float<T>(v.x)), to_float(from_float<T>(v.y)), to_float(from_float<T>(v.z)),
                     to_float(from_float<T>(v.w)));
}
__device__ __forceinline__ float4 mul4(float f, float4 x, float4 w) {
  return make_float4(f * x.x * w.x, f * x.y * w.y, f * x.z * w.z, f * x.w * w.w);
}
__device__ __forceinline__ float4 fma4v(float4 a, float4 x, float4 y) {
  return make_float4(fmaf(a.x, x.x, y.x), fmaf(a.y, x.y, y.y), fmaf(a.z, x.z, y.z), fmaf(a.w, x.w, y.w));
}

__device__ __forceinline__ float4 add4(float4 x, float4 y) { return make_float4(x.x + y.x, x.y + y.y, x.z + y.z, x.w + y.w); }

template <typename T, int THREADS, int NR, bool PLUS>
__global__ void __launch_bounds__(THREADS)
residual_step_vec_kernel(const b200_residual_step_args a) {
  __shared__ float red[THREADS / 32];
  __shared__ float unit[PLUS ? THREADS * NR : 1];  // squares of 4-column units, then a group's factor in its first one
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, nv = a.dim >> 2;
  const StepRow<T> row(a);
  float4 x[NR], y[NR];
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int i = tid + j * THREADS;
    x[j] = i < nv && !(PLUS && a.fresh) ? ld4f(row.x + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    y[j] = make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (row.y) {
    if (row.pw) {
#pragma unroll 4
      for (int k = 0; k < a.parts; ++k) {
        const float w = row.pw[k];
#pragma unroll
        for (int j = 0; j < NR; ++j) {
          const int i = tid + j * THREADS;
          if (i < nv) y[j] = fma4(w, load4(row.y + k * a.y_stride + 4 * i), y[j]);
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const int i = tid + j * THREADS;
        if (i < nv) y[j] = load4(row.y + 4 * i);
      }
    }
    if (row.extra)
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const int i = tid + j * THREADS;
        if (i < nv) y[j] = fma4(row.gate, load4(row.extra + 4 * i), y[j]);
      }
    if (PLUS && a.bias)
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const int i = tid + j * THREADS;
        if (i < nv) y[j] = add4(y[j], ld4f(a.bias + 4 * i));
      }
    if (!PLUS || a.out_norm) {
      float ss[1] = {0.f};
#pragma unroll
      for (int j = 0; j < NR; ++j) ss[0] += dot4(y[j]);
      block_sums<THREADS>(ss, red);
      const float f = 1.f / sqrtf(ss[0] / (float)a.dim + a.eps);
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const int i = tid + j * THREADS;
        if (i >= nv) continue;
        const float4 n = mul4(f, y[j], ld4f(a.out_norm + 4 * i));
        x[j] = make_float4(x[j].x + n.x, x[j].y + n.y, x[j].z + n.z, x[j].w + n.w);
        if (!PLUS && row.store) *reinterpret_cast<float4*>(row.x + 4 * i) = x[j];
      }
    } else {
#pragma unroll
      for (int j = 0; j < NR; ++j) x[j] = add4(x[j], y[j]);
    }
  }
  if (PLUS)
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int i = tid + j * THREADS;
      if (i >= nv) continue;
      if (row.embed) {
        const float4 e = load4(row.embed + 4 * i);  // the scaled row is rounded before it is added, as where it starts a stream
        x[j] = make_float4(x[j].x + __fmul_rn(a.table_scale, e.x), x[j].y + __fmul_rn(a.table_scale, e.y),
                           x[j].z + __fmul_rn(a.table_scale, e.z), x[j].w + __fmul_rn(a.table_scale, e.w));
      }
      if (a.add) x[j] = add4(x[j], ld4f(a.add + 4 * i));
      if (row.store && (row.y || a.table || a.add)) *reinterpret_cast<float4*>(row.x + 4 * i) = x[j];
    }
  if (!row.h && !(PLUS && row.h32)) return;
  float f;
  int per = 1;  // 4-column units of a group
  if (PLUS && a.groups > 1) {
    per = nv / a.groups;
#pragma unroll
    for (int j = 0; j < NR; ++j)
      if (tid + j * THREADS < nv) unit[tid + j * THREADS] = dot4(x[j]);
    __syncthreads();
    for (int g = tid >> 5; g < a.groups; g += THREADS / 32) {
      float part = 0.f;
      for (int u = tid & 31; u < per; u += 32) part += unit[g * per + u];
      part = warp_sum(part);
      if ((tid & 31) == 0) unit[g * per] = 1.f / sqrtf(part / (float)(4 * per) + a.eps);
    }
    __syncthreads();
  } else {
    float ss[1] = {0.f};
#pragma unroll
    for (int j = 0; j < NR; ++j) ss[0] += dot4(x[j]);
    block_sums<THREADS>(ss, red);
    f = 1.f / sqrtf(ss[0] / (float)a.dim + a.eps);
  }
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int i = tid + j * THREADS;
    if (i >= nv) continue;
    if (PLUS && a.groups > 1) f = unit[i / per * per];
    float4 h = mul4(f, x[j], ld4f(a.in_norm + 4 * i));
    if (PLUS && row.h32) {
      *reinterpret_cast<float4*>(row.h32 + 4 * i) = h;
      continue;
    }
    if (PLUS && a.mixes > 0) {
      const float4 v = row.seen > 0 ? ld4f(row.last + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 d = make_float4(v.x - h.x, v.y - h.y, v.z - h.z, v.w - h.w);
      for (int k = 0; k < a.mixes; ++k)
        store4(row.h + k * a.mix_stride + 4 * i, fma4v(d, ld4f(a.mix_weight + (int64_t)k * a.dim + 4 * i), h));
      *reinterpret_cast<float4*>(row.last + 4 * i) = h;
      continue;
    }
    if (a.conv_weight) {
      h = round4<T>(h);  // what the slot keeps
      const int older = a.taps - 1;
      float4 acc = fma4v(ld4f(a.conv_weight + (int64_t)older * a.dim + 4 * i), h, h);
      for (int k = 0; k < older; ++k) {  // oldest first; the slot moves up by one on the way
        const float4 v = row.seen >= older - k ? load4(row.state + (int64_t)k * a.dim + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        acc = fma4v(ld4f(a.conv_weight + (int64_t)k * a.dim + 4 * i), v, acc);
        if (k > 0) store4(row.state + (int64_t)(k - 1) * a.dim + 4 * i, v);
      }
      if (older > 0) store4(row.state + (int64_t)(older - 1) * a.dim + 4 * i, h);
      h = acc;
    }
    store4(row.h + 4 * i, h);
  }
}

// Any width: the row waits in shared memory for its norms.
template <typename T>
__global__ void __launch_bounds__(256)
residual_step_kernel(const b200_residual_step_args a) {
  extern __shared__ float u[];
  __shared__ float red[8];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, dim = a.dim;
  const StepRow<T> row(a);
  float ss[1] = {0.f};
  const bool changes = row.y || a.table || a.add;
  auto plus = [&](int d, float x) {
    if (row.embed) x += __fmul_rn(a.table_scale, to_float(row.embed[d]));
    if (a.add) x += a.add[d];
    if (row.store && changes) row.x[d] = x;
    u[d] = x;
    ss[0] += x * x;
  };
  if (row.y) {
    for (int d = tid; d < dim; d += 256) {
      float y = 0.f;
      if (row.pw) {
        for (int k = 0; k < a.parts; ++k) y = fmaf(row.pw[k], to_float(row.y[k * a.y_stride + d]), y);
      } else {
        y = to_float(row.y[d]);
      }
      if (row.extra) y = fmaf(row.gate, to_float(row.extra[d]), y);
      if (a.bias) y += a.bias[d];
      u[d] = y;
      ss[0] += y * y;
    }
    float f = 1.f;
    if (a.out_norm) {
      block_sums<256>(ss, red);
      f = 1.f / sqrtf(ss[0] / (float)dim + a.eps);
    }
    ss[0] = 0.f;
    for (int d = tid; d < dim; d += 256) {
      const float r = a.out_norm ? f * u[d] * a.out_norm[d] : u[d];
      plus(d, (a.fresh ? 0.f : row.x[d]) + r);
    }
  } else {
    for (int d = tid; d < dim; d += 256) plus(d, a.fresh ? 0.f : row.x[d]);
  }
  if (!row.h && !row.h32) return;
  const int groups = a.groups > 1 ? a.groups : 1, size = dim / groups;
  float f = 1.f;
  if (groups == 1) {
    block_sums<256>(ss, red);
    f = 1.f / sqrtf(ss[0] / (float)dim + a.eps);
  } else {  // a warp per group: its columns are divided where they are
    __syncthreads();
    for (int g = tid >> 5; g < groups; g += 8) {
      float part = 0.f;
      for (int d = tid & 31; d < size; d += 32) part += u[g * size + d] * u[g * size + d];
      part = 1.f / sqrtf(warp_sum(part) / (float)size + a.eps);
      for (int d = tid & 31; d < size; d += 32) u[g * size + d] *= part;
    }
    __syncthreads();
  }
  for (int d = tid; d < dim; d += 256) {
    float h = f * u[d] * a.in_norm[d];
    if (row.h32) {
      row.h32[d] = h;
      continue;
    }
    if (a.mixes > 0) {
      const float v = row.seen > 0 ? row.last[d] : 0.f;
      for (int k = 0; k < a.mixes; ++k) row.h[k * a.mix_stride + d] = from_float<T>(fmaf(v - h, a.mix_weight[(int64_t)k * dim + d], h));
      row.last[d] = h;
      continue;
    }
    if (a.conv_weight) {
      h = to_float(from_float<T>(h));
      const int older = a.taps - 1;
      float acc = fmaf(a.conv_weight[(int64_t)older * dim + d], h, h);
      for (int k = 0; k < older; ++k) {
        const float v = row.seen >= older - k ? to_float(row.state[(int64_t)k * dim + d]) : 0.f;
        acc = fmaf(a.conv_weight[(int64_t)k * dim + d], v, acc);
        if (k > 0) row.state[(int64_t)(k - 1) * dim + d] = from_float<T>(v);
      }
      if (older > 0) row.state[(int64_t)(older - 1) * dim + d] = from_float<T>(h);
      h = acc;
    }
    row.h[d] = from_float<T>(h);
  }
}

constexpr int kMaxGenericStepDim = 48 * 1024;  // fp32 columns of one row in shared memory

inline bool plus_form(const b200_residual_step_args& a) {
  return (a.y && !a.out_norm) || a.bias || a.table || a.add || a.h32 || a.mixes > 0 || a.groups > 1 || a.fresh;
}

template <typename T, int THREADS, int NR>
int launch_step_form(const b200_residual_step_args& a, cudaStream_t st) {
  auto* kern = plus_form(a) ? residual_step_vec_kernel<T, THREADS, NR, true> : residual_step_vec_kernel<T, THREADS, NR, false>;
  B200_CUDA_OK(launch_pdl(kern, dim3(a.rows), dim3(THREADS), 0, st, a));
  return check_launch("residual_step");
}

template <typename T>
int launch_residual_step(const b200_residual_step_args& a, cudaStream_t st) {
  auto ok = [](const void* p, int64_t stride, int size) {
    return !p || ((uintptr_t)p % (4 * size) == 0 && stride % 4 == 0);
  };
  const bool vec = a.dim % 4 == 0 && a.dim <= 8192 && ok(a.x, 4, 4) && ok(a.y, a.y_stride, sizeof(T)) &&
                   ok(a.extra, a.extra_stride, sizeof(T)) && ok(a.h, a.h_stride, sizeof(T)) && ok(a.state, 4, sizeof(T)) &&
                   ok(a.out_norm, 4, 4) && ok(a.in_norm, 4, 4) && ok(a.conv_weight, 4, 4) && ok(a.bias, 4, 4) &&
                   ok(a.table, 4, sizeof(T)) && ok(a.add, 4, 4) && ok(a.h32, a.h_stride, 4) && ok(a.mix_weight, a.mix_stride, 4) &&
                   ok(a.mix_state, 4, 4) && (a.groups <= 1 || a.dim % (4 * a.groups) == 0);
  if (vec) {
    // two 4-column units a thread where the machine is full; with few rows the latency of one counts
    const int nv = a.dim / 4;
    const bool few = a.rows <= 2 * sm_count();
    if (nv <= 64) return launch_step_form<T, 64, 1>(a, st);
    if (nv <= 128) return launch_step_form<T, 128, 1>(a, st);
    if (nv <= 256) return launch_step_form<T, 256, 1>(a, st);
    if (nv <= 512) return few ? launch_step_form<T, 512, 1>(a, st) : launch_step_form<T, 256, 2>(a, st);
    if (nv <= 768) return few ? launch_step_form<T, 1024, 1>(a, st) : launch_step_form<T, 384, 2>(a, st);
    if (nv <= 1024) return few ? launch_step_form<T, 1024, 1>(a, st) : launch_step_form<T, 512, 2>(a, st);
    return launch_step_form<T, 512, 4>(a, st);
  }
  const size_t smem = (size_t)a.dim * sizeof(float);
  static size_t attr = 0;  // per instantiation: what was asked for so far
  if (smem > 32 * 1024 && smem > attr) {
    B200_CUDA_OK(cudaFuncSetAttribute(residual_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attr = smem;
  }
  B200_CUDA_OK(launch_pdl(residual_step_kernel<T>, dim3(a.rows), dim3(256), smem, st, a));
  return check_launch("residual_step");
}

// ---- token mixes of portions -----------------------------------------------------------------------
// A thread walks kMixTile rows of its columns with the row before in registers; only the first tile of a segment touches the
// slot, and it takes the segment's last row straight from the input, so the tiles never race.
constexpr int kMixTile = 8;

template <typename T, int MIXES>  // 4 columns a thread; MIXES = 0: as many as a.mixes says
__global__ void __launch_bounds__(128)
token_mix_vec_kernel(const float* h, const float* weight, float* state, const int32_t* cu, const int32_t* seq_lens,
                     const int32_t* slots, T* out, int dim, int mixes_rt, int64_t h_stride, int64_t out_stride, int64_t mix_stride) {
  pdl_trigger();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4, mixes = MIXES > 0 ? MIXES : mixes_rt;
  float4 w[MIXES > 0 ? MIXES : 1];
  if (MIXES > 0 && c < dim)
#pragma unroll
    for (int k = 0; k < MIXES; ++k) w[k] = ld4f(weight + (int64_t)k * dim + c);
  pdl_wait();
  const int s = blockIdx.y, row0 = cu[s], len = cu[s + 1] - row0, t0 = blockIdx.z * kMixTile;
  if (t0 >= len || c >= dim) return;
  float* st = state + (int64_t)slots[s] * dim + c;
  const float* x = h + (int64_t)row0 * h_stride + c;
  float4 last = make_float4(0.f, 0.f, 0.f, 0.f);
  if (t0 > 0)
    last = ld4f(x + (int64_t)(t0 - 1) * h_stride);
  else if (seq_lens[s] != len)
    last = ld4f(st);
  if (t0 == 0) *reinterpret_cast<float4*>(st) = ld4f(x + (int64_t)(len - 1) * h_stride);
  const int n = min(kMixTile, len - t0);
  float4 rows[kMixTile];
#pragma unroll
  for (int i = 0; i < kMixTile; ++i)
    if (i < n) rows[i] = ld4f(x + (int64_t)(t0 + i) * h_stride);
#pragma unroll
  for (int i = 0; i < kMixTile; ++i) {
    if (i >= n) break;
    const float4 v = rows[i], d = make_float4(last.x - v.x, last.y - v.y, last.z - v.z, last.w - v.w);
    T* o = out + (int64_t)(row0 + t0 + i) * out_stride + c;
#pragma unroll
    for (int k = 0; k < (MIXES > 0 ? MIXES : B200_MAX_MIXES); ++k) {
      if (k >= mixes) break;
      store4(o + k * mix_stride, fma4v(d, MIXES > 0 ? w[MIXES > 0 ? k : 0] : ld4f(weight + (int64_t)k * dim + c), v));
    }
    last = v;
  }
}

template <typename T>  // any width
__global__ void __launch_bounds__(128)
token_mix_kernel(const float* h, const float* weight, float* state, const int32_t* cu, const int32_t* seq_lens,
                 const int32_t* slots, T* out, int dim, int mixes, int64_t h_stride, int64_t out_stride, int64_t mix_stride) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * 128 + threadIdx.x;
  const int s = blockIdx.y, row0 = cu[s], len = cu[s + 1] - row0, t0 = blockIdx.z * kMixTile;
  if (t0 >= len || c >= dim) return;
  float* st = state + (int64_t)slots[s] * dim + c;
  const float* x = h + (int64_t)row0 * h_stride + c;
  float last = t0 > 0 ? x[(int64_t)(t0 - 1) * h_stride] : seq_lens[s] != len ? *st : 0.f;
  if (t0 == 0) *st = x[(int64_t)(len - 1) * h_stride];
  for (int t = t0; t < min(t0 + kMixTile, len); ++t) {
    const float v = x[(int64_t)t * h_stride];
    for (int k = 0; k < mixes; ++k)
      out[k * mix_stride + (int64_t)(row0 + t) * out_stride + c] = from_float<T>(fmaf(last - v, weight[(int64_t)k * dim + c], v));
    last = v;
  }
}

}  // namespace
}  // namespace b200

extern "C" int b200_token_mix(const float* h, const float* weight, float* state, const int32_t* cu_seqlens,
                              const int32_t* seq_lens, const int32_t* slots, void* out, int num_seqs, int max_q_len, int dim,
                              int mixes, int64_t h_stride, int64_t out_stride, int64_t mix_stride, int dtype, void* stream) {
  using namespace b200;
  B200_CHECK_ARG(h && weight && state && cu_seqlens && seq_lens && slots && out && dim > 0, "token_mix: bad arguments");
  B200_CHECK_ARG(mixes >= 1 && mixes <= B200_MAX_MIXES, "token_mix: %d mixes (at most %d)", mixes, B200_MAX_MIXES);
  if (num_seqs <= 0 || max_q_len <= 0) return B200_OK;
  const int tiles = (max_q_len + kMixTile - 1) / kMixTile;
  B200_CHECK_ARG(num_seqs <= 65535 && tiles <= 65535, "token_mix: batch too large");
  return B200_DISPATCH_DTYPE(dtype, T, [&]() -> int {
    const bool vec = dim % 4 == 0 && h_stride % 4 == 0 && out_stride % 4 == 0 && mix_stride % 4 == 0 &&
                     (((uintptr_t)h | (uintptr_t)weight | (uintptr_t)state) & 15) == 0 && (uintptr_t)out % (4 * sizeof(T)) == 0;
    auto* kern = !vec ? token_mix_kernel<T> : mixes == 5 ? token_mix_vec_kernel<T, 5> : token_mix_vec_kernel<T, 0>;
    const int cols = vec ? 512 : 128;
    B200_CUDA_OK(launch_pdl(kern, dim3((dim + cols - 1) / cols, num_seqs, tiles), dim3(128), 0, (cudaStream_t)stream, h, weight,
                            state, cu_seqlens, seq_lens, slots, (T*)out, dim, mixes, h_stride, out_stride, mix_stride));
    return check_launch("token_mix");
  });
}

extern "C" int b200_residual_step(const b200_residual_step_args* a, void* stream) {
  using namespace b200;
  B200_CHECK_ARG(a && a->x && (a->y || a->h || a->h32 || a->table || a->add), "residual_step: nothing to do");
  B200_CHECK_ARG(a->dim >= 1 && a->dim <= kMaxGenericStepDim, "residual_step: width %d outside 1..%d", a->dim, kMaxGenericStepDim);
  B200_CHECK_ARG(a->parts >= 0 && (a->parts == 0 || (a->y && a->part_weight)), "residual_step: parts without weights");
  B200_CHECK_ARG(!a->extra || (a->y && a->extra_gate), "residual_step: a shared part without its gate");
  B200_CHECK_ARG(!(a->h || a->h32) || a->in_norm, "residual_step: an input without its norm");
  B200_CHECK_ARG(!a->bias || a->y, "residual_step: a bias without its result");
  B200_CHECK_ARG(!a->table || (a->ids && a->vocab > 0), "residual_step: embedding rows without ids");
  B200_CHECK_ARG(!a->fresh || a->table, "residual_step: a fresh stream without embedding rows");
  B200_CHECK_ARG(a->groups >= 0 && (a->groups <= 1 || a->dim % a->groups == 0), "residual_step: %d columns in %d groups", a->dim,
                 a->groups);
  B200_CHECK_ARG(a->mixes == 0 || (a->mixes >= 1 && a->mixes <= B200_MAX_MIXES && a->h && !a->h32 && !a->conv_weight && !a->row_ids &&
                                   a->mix_weight && a->mix_state && a->slots && a->seq_lens),
                 "residual_step: %d mixes without their state", a->mixes);
  B200_CHECK_ARG(!a->h32 || (!a->h && !a->conv_weight), "residual_step: a 32-bit input stands alone");
  B200_CHECK_ARG(!a->conv_weight || (a->h && a->taps >= 1 && a->taps <= kMaxStepTaps && a->seq_lens && !a->row_ids &&
                                     (a->taps == 1 || (a->state && a->slots))),
                 "residual_step: a convolution of %d taps without its state", a->taps);
  if (a->rows <= 0) return B200_OK;
  return B200_DISPATCH_DTYPE(a->dtype, T, [&]() -> int { return launch_residual_step<T>(*a, (cudaStream_t)stream); });
}
