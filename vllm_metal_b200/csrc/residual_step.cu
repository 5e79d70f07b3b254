// The step between two sublayers that stand between norms of their own (include/b200_hybrid_ops.h): the result's norm,
// the sum, the next input's norm and, for single rows, the short convolution on that input, in one launch.  A result may
// arrive as the weighted parts of routed experts and a gated shared part.
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
    seen = a.conv_weight ? a.seq_lens[b] - 1 : 0;
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

template <typename T, int THREADS, int NR>
__global__ void __launch_bounds__(THREADS)
residual_step_vec_kernel(const b200_residual_step_args a) {
  __shared__ float red[THREADS / 32];
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x, nv = a.dim >> 2;
  const StepRow<T> row(a);
  float4 x[NR], y[NR];
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int i = tid + j * THREADS;
    x[j] = i < nv ? ld4f(row.x + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
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
      if (row.store) *reinterpret_cast<float4*>(row.x + 4 * i) = x[j];
    }
  }
  if (!row.h) return;
  float ss[1] = {0.f};
#pragma unroll
  for (int j = 0; j < NR; ++j) ss[0] += dot4(x[j]);
  block_sums<THREADS>(ss, red);
  const float f = 1.f / sqrtf(ss[0] / (float)a.dim + a.eps);
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int i = tid + j * THREADS;
    if (i >= nv) continue;
    float4 h = mul4(f, x[j], ld4f(a.in_norm + 4 * i));
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
  if (row.y) {
    for (int d = tid; d < dim; d += 256) {
      float y = 0.f;
      if (row.pw) {
        for (int k = 0; k < a.parts; ++k) y = fmaf(row.pw[k], to_float(row.y[k * a.y_stride + d]), y);
      } else {
        y = to_float(row.y[d]);
      }
      if (row.extra) y = fmaf(row.gate, to_float(row.extra[d]), y);
      u[d] = y;
      ss[0] += y * y;
    }
    block_sums<256>(ss, red);
    const float f = 1.f / sqrtf(ss[0] / (float)dim + a.eps);
    ss[0] = 0.f;
    for (int d = tid; d < dim; d += 256) {
      const float x = row.x[d] + f * u[d] * a.out_norm[d];
      if (row.store) row.x[d] = x;
      u[d] = x;
      ss[0] += x * x;
    }
  } else {
    for (int d = tid; d < dim; d += 256) {
      u[d] = row.x[d];
      ss[0] += u[d] * u[d];
    }
  }
  if (!row.h) return;
  block_sums<256>(ss, red);
  const float f = 1.f / sqrtf(ss[0] / (float)dim + a.eps);
  for (int d = tid; d < dim; d += 256) {
    float h = f * u[d] * a.in_norm[d];
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

template <typename T, int THREADS, int NR>
int launch_step_form(const b200_residual_step_args& a, cudaStream_t st) {
  B200_CUDA_OK(launch_pdl(residual_step_vec_kernel<T, THREADS, NR>, dim3(a.rows), dim3(THREADS), 0, st, a));
  return check_launch("residual_step");
}

template <typename T>
int launch_residual_step(const b200_residual_step_args& a, cudaStream_t st) {
  auto ok = [](const void* p, int64_t stride, int size) {
    return !p || ((uintptr_t)p % (4 * size) == 0 && stride % 4 == 0);
  };
  const bool vec = a.dim % 4 == 0 && a.dim <= 8192 && ok(a.x, 4, 4) && ok(a.y, a.y_stride, sizeof(T)) &&
                   ok(a.extra, a.extra_stride, sizeof(T)) && ok(a.h, a.h_stride, sizeof(T)) && ok(a.state, 4, sizeof(T)) &&
                   ok(a.out_norm, 4, 4) && ok(a.in_norm, 4, 4) && ok(a.conv_weight, 4, 4);
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

}  // namespace
}  // namespace b200

extern "C" int b200_residual_step(const b200_residual_step_args* a, void* stream) {
  using namespace b200;
  B200_CHECK_ARG(a && a->x && (a->y || a->h), "residual_step: nothing to do");
  B200_CHECK_ARG(a->dim >= 1 && a->dim <= kMaxGenericStepDim, "residual_step: width %d outside 1..%d", a->dim, kMaxGenericStepDim);
  B200_CHECK_ARG(!a->y || a->out_norm, "residual_step: a result without its norm");
  B200_CHECK_ARG(a->parts >= 0 && (a->parts == 0 || (a->y && a->part_weight)), "residual_step: parts without weights");
  B200_CHECK_ARG(!a->extra || (a->y && a->extra_gate), "residual_step: a shared part without its gate");
  B200_CHECK_ARG(!a->h || a->in_norm, "residual_step: an input without its norm");
  B200_CHECK_ARG(!a->conv_weight || (a->h && a->taps >= 1 && a->taps <= kMaxStepTaps && a->seq_lens && !a->row_ids &&
                                     (a->taps == 1 || (a->state && a->slots))),
                 "residual_step: a convolution of %d taps without its state", a->taps);
  if (a->rows <= 0) return B200_OK;
  return B200_DISPATCH_DTYPE(a->dtype, T, [&]() -> int { return launch_residual_step<T>(*a, (cudaStream_t)stream); });
}
