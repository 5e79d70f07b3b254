// The hyper-connected residual between sublayers (include/b200_hybrid_ops.h): several fp32 copies of the stream, read
// through one vector of weights, written back through a mixing matrix.
//
// Everything between the products of one sublayer and those of the next is one launch: norms of the result's halves,
// residual gate, mixing, the next sublayer's combination and its layer norm, at decode also the token shift.  HBM-bound at
// 2 * num_streams * dim * 4 bytes a row plus the 16-bit operands; one CTA a row, the combined row in registers.
#include "../../include/b200_hybrid_ops.h"
#include "row_ops.cuh"

namespace b200 {
namespace {

// ---- embedding ------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
embed_streams_kernel(const int32_t* __restrict__ ids, const T* __restrict__ table, const int32_t* __restrict__ positions,
                     const float* __restrict__ freq, float* __restrict__ out, int vocab, int dim, int streams) {
  pdl_trigger();
  pdl_wait();
  const int id = ids[blockIdx.x];
  const float p = positions ? (float)positions[blockIdx.x] : 0.f;
  float* o = out + (int64_t)blockIdx.x * streams * dim;
  const bool ok = id >= 0 && id < vocab;
  for (int i = threadIdx.x; 2 * i < dim; i += 256) {
    float v[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) v[e] = ok && 2 * i + e < dim ? to_float(table[(int64_t)id * dim + 2 * i + e]) : 0.f;
    if (positions) {
      // what the rounded product and the frequency's low part leave of the angle, r, turns it by a few Taylor terms
      const float hi = freq[2 * i], a = p * hi, r = fmaf(p, freq[2 * i + 1], fmaf(p, hi, -a));
      float sn, cs;
      sincosf(a, &sn, &cs);
      const float s1 = fmaf(-r * r, r * (1.f / 6.f), r), c1 = -0.5f * r * r;  // sin r, cos r - 1
      v[0] += sn + fmaf(s1, cs, c1 * sn);
      v[1] += cs + fmaf(-s1, sn, c1 * cs);
    }
    for (int s = 0; s < streams; ++s) {
      o[(int64_t)s * dim + 2 * i] = v[0];
      if (2 * i + 1 < dim) o[(int64_t)s * dim + 2 * i + 1] = v[1];
    }
  }
}

// ---- the step between two sublayers ---------------------------------------------------------------
template <typename T>
struct Row {  // pointers of one row
  const T *y, *y2, *gate;
  float* x;
  T *h, *shifted, *prev;
  bool fresh;
  __device__ Row(const b200_stream_step_args& a) {
    const int64_t b = blockIdx.x, r = a.row_ids ? a.row_ids[b] : b;
    x = a.streams + r * a.num_streams * a.dim;
    y = a.y ? reinterpret_cast<const T*>(a.y) + r * a.y_stride : nullptr;
    y2 = a.y2 ? reinterpret_cast<const T*>(a.y2) + r * a.y2_stride : nullptr;
    gate = a.gate ? reinterpret_cast<const T*>(a.gate) + r * a.gate_stride : nullptr;
    h = a.h ? reinterpret_cast<T*>(a.h) + b * a.h_stride : nullptr;
    shifted = a.shifted ? reinterpret_cast<T*>(a.shifted) + b * a.shifted_stride : nullptr;
    prev = a.shifted ? reinterpret_cast<T*>(a.previous) + (int64_t)a.slots[b] * a.dim : nullptr;
    fresh = a.shifted ? a.seq_lens[b] == 1 : true;
  }
};

template <typename T, int S, int THREADS, int NR>
__global__ void __launch_bounds__(THREADS)
stream_step_vec_kernel(const b200_stream_step_args a) {
  __shared__ float red[2 * THREADS / 32];
  __shared__ float mix[S * S], outw[S], inw[S];
  pdl_trigger();
  const int tid = threadIdx.x, dim = a.dim, nv = dim >> 2;
  if (tid < S * S) mix[tid] = a.y ? a.mix[tid] : 0.f;  // weights: nothing earlier in the stream writes them
  if (tid < S) {
    outw[tid] = a.y ? a.out_weight[tid] : 0.f;
    inw[tid] = a.h ? a.in_weight[tid] : 0.f;
  }
  pdl_wait();
  __syncthreads();
  const Row<T> row(a);
  float4 y[NR];
  if (row.y) {
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int i = tid + j * THREADS;
      y[j] = i < nv ? load4(row.y + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (row.y2) {
      float4 z[NR];
      float ss[2] = {0.f, 0.f};
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const int i = tid + j * THREADS;
        z[j] = i < nv ? load4(row.y2 + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        ss[0] += dot4(y[j]);
        ss[1] += dot4(z[j]);
      }
      block_sums<THREADS>(ss, red);
      const float fy = 0.5f / sqrtf(ss[0] / (float)dim + a.eps), fz = 0.5f / sqrtf(ss[1] / (float)dim + a.eps);
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const int i = tid + j * THREADS;
        if (i >= nv) continue;
        const float4 wy = ld4f(a.y_norm + 4 * i), wz = ld4f(a.y2_norm + 4 * i);
        y[j] = make_float4(y[j].x * fy * wy.x + z[j].x * fz * wz.x, y[j].y * fy * wy.y + z[j].y * fz * wz.y,
                           y[j].z * fy * wy.z + z[j].z * fz * wz.z, y[j].w * fy * wy.w + z[j].w * fz * wz.w);
      }
    }
    if (row.gate) {
#pragma unroll
      for (int j = 0; j < NR; ++j) {
        const int i = tid + j * THREADS;
        if (i >= nv) continue;
        const float4 g = load4(row.gate + 4 * i), b = ld4f(a.gate_bias + 4 * i);
        y[j].x *= gate_f(g.x + b.x);
        y[j].y *= gate_f(g.y + b.y);
        y[j].z *= gate_f(g.z + b.z);
        y[j].w *= gate_f(g.w + b.w);
      }
    }
  }
  float4 u[NR];
  float sum[1] = {0.f};
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int i = tid + j * THREADS;
    u[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= nv) continue;
    float4 x[S];
#pragma unroll
    for (int s = 0; s < S; ++s) x[s] = ld4f(row.x + s * dim + 4 * i);
    if (row.y) {
      float4 n[S];
#pragma unroll
      for (int t = 0; t < S; ++t) {
        n[t] = make_float4(outw[t] * y[j].x, outw[t] * y[j].y, outw[t] * y[j].z, outw[t] * y[j].w);
#pragma unroll
        for (int s = 0; s < S; ++s) n[t] = fma4(mix[s * S + t], x[s], n[t]);
      }
#pragma unroll
      for (int t = 0; t < S; ++t) {
        x[t] = n[t];
        if (a.store) *reinterpret_cast<float4*>(row.x + t * dim + 4 * i) = n[t];
      }
    }
#pragma unroll
    for (int s = 0; s < S; ++s) u[j] = fma4(inw[s], x[s], u[j]);
    sum[0] += u[j].x + u[j].y + u[j].z + u[j].w;
  }
  if (!row.h) return;
  block_sums<THREADS>(sum, red);
  const float mean = sum[0] / (float)dim;
  float var[1] = {0.f};
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    if (tid + j * THREADS >= nv) continue;
    u[j] = make_float4(u[j].x - mean, u[j].y - mean, u[j].z - mean, u[j].w - mean);
    var[0] += dot4(u[j]);
  }
  block_sums<THREADS>(var, red);
  const float inv = 1.f / sqrtf(var[0] / (float)dim + a.eps);
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int i = tid + j * THREADS;
    if (i >= nv) continue;
    const float4 w = ld4f(a.norm_weight + 4 * i);
    const float4 h = make_float4(u[j].x * inv * w.x, u[j].y * inv * w.y, u[j].z * inv * w.z, u[j].w * inv * w.w);
    store4(row.h + 4 * i, h);
    if (row.shifted) {
      const float4 sh = ld4f(a.shift + 4 * i);
      const float4 p = row.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(row.prev + 4 * i);
      store4(row.prev + 4 * i, h);
      store4(row.shifted + 4 * i, make_float4(fmaf(p.x - h.x, sh.x, h.x), fmaf(p.y - h.y, sh.y, h.y),
                                              fmaf(p.z - h.z, sh.z, h.z), fmaf(p.w - h.w, sh.w, h.w)));
    }
  }
}

// Any number of streams and any width: the combined row waits in shared memory for its norm.
template <typename T>
__global__ void __launch_bounds__(256)
stream_step_kernel(const b200_stream_step_args a) {
  extern __shared__ float u[];
  __shared__ float red[2 * 256 / 32];
  __shared__ float mix[B200_MAX_STREAMS * B200_MAX_STREAMS], outw[B200_MAX_STREAMS], inw[B200_MAX_STREAMS];
  pdl_trigger();
  const int tid = threadIdx.x, dim = a.dim, S = a.num_streams;
  if (tid < S * S) mix[tid] = a.y ? a.mix[tid] : 0.f;
  if (tid < S) {
    outw[tid] = a.y ? a.out_weight[tid] : 0.f;
    inw[tid] = a.h ? a.in_weight[tid] : 0.f;
  }
  pdl_wait();
  __syncthreads();
  const Row<T> row(a);
  float fy = 1.f, fz = 0.f;
  if (row.y2) {
    float ss[2] = {0.f, 0.f};
    for (int d = tid; d < dim; d += 256) {
      const float y = to_float(row.y[d]), z = to_float(row.y2[d]);
      ss[0] += y * y;
      ss[1] += z * z;
    }
    block_sums<256>(ss, red);
    fy = 0.5f / sqrtf(ss[0] / (float)dim + a.eps);
    fz = 0.5f / sqrtf(ss[1] / (float)dim + a.eps);
  }
  float sum[1] = {0.f};
  for (int d = tid; d < dim; d += 256) {
    float x[B200_MAX_STREAMS];
    for (int s = 0; s < S; ++s) x[s] = row.x[(int64_t)s * dim + d];
    float c = 0.f;
    if (row.y) {
      float y = to_float(row.y[d]);
      if (row.y2) y = y * fy * a.y_norm[d] + to_float(row.y2[d]) * fz * a.y2_norm[d];
      if (row.gate) y *= gate_f(to_float(row.gate[d]) + a.gate_bias[d]);
      for (int t = 0; t < S; ++t) {
        float n = outw[t] * y;
        for (int s = 0; s < S; ++s) n = fmaf(mix[s * S + t], x[s], n);
        if (a.store) row.x[(int64_t)t * dim + d] = n;
        c = fmaf(inw[t], n, c);
      }
    } else {
      for (int s = 0; s < S; ++s) c = fmaf(inw[s], x[s], c);
    }
    u[d] = c;
    sum[0] += c;
  }
  if (!row.h) return;
  block_sums<256>(sum, red);
  const float mean = sum[0] / (float)dim;
  float var[1] = {0.f};
  for (int d = tid; d < dim; d += 256) var[0] += (u[d] - mean) * (u[d] - mean);
  block_sums<256>(var, red);
  const float inv = 1.f / sqrtf(var[0] / (float)dim + a.eps);
  for (int d = tid; d < dim; d += 256) {
    const float h = (u[d] - mean) * inv * a.norm_weight[d];
    row.h[d] = from_float<T>(h);
    if (row.shifted) {
      const float p = row.fresh ? 0.f : to_float(row.prev[d]);
      row.prev[d] = from_float<T>(h);
      row.shifted[d] = from_float<T>(fmaf(p - h, a.shift[d], h));
    }
  }
}

constexpr int kMaxGenericDim = 48 * 1024;  // fp32 columns of one row in shared memory

template <typename T, int S, int THREADS, int NR>
int launch_form(const b200_stream_step_args& a, cudaStream_t st) {
  B200_CUDA_OK(launch_pdl(stream_step_vec_kernel<T, S, THREADS, NR>, dim3(a.rows), dim3(THREADS), 0, st, a));
  return check_launch("stream_step");
}

// Two 4-column units a thread measured fastest where the machine is full; with few rows the latency of one counts.
template <typename T, int S>
int launch_vec(const b200_stream_step_args& a, cudaStream_t st) {
  const int nv = a.dim / 4;
  if (nv <= 64) return launch_form<T, S, 64, 1>(a, st);
  if (nv <= 128) return launch_form<T, S, 128, 1>(a, st);
  if (nv <= 256) return launch_form<T, S, 256, 1>(a, st);
  if (a.rows <= 2 * sm_count() && nv <= 1024)
    return nv <= 512 ? launch_form<T, S, 512, 1>(a, st) : launch_form<T, S, 1024, 1>(a, st);
  if (nv <= 512) return launch_form<T, S, 256, 2>(a, st);
  if (nv <= 640) return launch_form<T, S, 320, 2>(a, st);
  if (nv <= 768) return launch_form<T, S, 384, 2>(a, st);
  if (nv <= 1024) return launch_form<T, S, 512, 2>(a, st);
  return launch_form<T, S, 512, 4>(a, st);
}

template <typename T>
int launch_step(const b200_stream_step_args& a, cudaStream_t st) {
  auto ok = [](const void* p, int64_t stride, int size) {
    return !p || ((uintptr_t)p % (4 * size) == 0 && stride % 4 == 0);
  };
  const bool vec = a.dim % 4 == 0 && a.dim <= 8192 && ok(a.streams, 4, 4) && ok(a.y, a.y_stride, sizeof(T)) &&
                   ok(a.y2, a.y2_stride, sizeof(T)) && ok(a.gate, a.gate_stride, sizeof(T)) &&
                   ok(a.h, a.h_stride, sizeof(T)) && ok(a.shifted, a.shifted_stride, sizeof(T)) &&
                   ok(a.previous, 4, sizeof(T)) && ok(a.y_norm, 4, 4) && ok(a.y2_norm, 4, 4) && ok(a.gate_bias, 4, 4) &&
                   ok(a.norm_weight, 4, 4) && ok(a.shift, 4, 4);
  if (vec) switch (a.num_streams) {
      case 1: return launch_vec<T, 1>(a, st);
      case 2: return launch_vec<T, 2>(a, st);
      case 3: return launch_vec<T, 3>(a, st);
      case 4: return launch_vec<T, 4>(a, st);
      default: break;
    }
  const size_t smem = (size_t)a.dim * sizeof(float);
  static int attr = 0;  // per instantiation: what was asked for so far
  if (smem > 32 * 1024 && (int)smem > attr) {
    B200_CUDA_OK(cudaFuncSetAttribute(stream_step_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    attr = (int)smem;
  }
  B200_CUDA_OK(launch_pdl(stream_step_kernel<T>, dim3(a.rows), dim3(256), smem, st, a));
  return check_launch("stream_step");
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_embed_streams(const int32_t* ids, const void* table, const int32_t* positions, const float* freq, float* out,
                       int rows, int vocab, int dim, int num_streams, int dtype, void* stream) {
  B200_CHECK_ARG(ids && table && out && vocab > 0 && dim > 0 && num_streams > 0, "embed_streams: bad arguments");
  B200_CHECK_ARG(!positions || freq, "embed_streams: positions without frequencies");
  if (rows <= 0) return B200_OK;
  return B200_DISPATCH_DTYPE(dtype, T, [&]() -> int {
    B200_CUDA_OK(launch_pdl(embed_streams_kernel<T>, dim3(rows), dim3(256), 0, (cudaStream_t)stream, ids,
                            (const T*)table, positions, freq, out, vocab, dim, num_streams));
    return check_launch("embed_streams");
  });
}

int b200_stream_step(const b200_stream_step_args* a, void* stream) {
  B200_CHECK_ARG(a && a->streams && (a->y || a->h), "stream_step: nothing to do");
  B200_CHECK_ARG(a->num_streams >= 1 && a->num_streams <= B200_MAX_STREAMS, "stream_step: %d streams outside 1..%d",
                 a->num_streams, B200_MAX_STREAMS);
  B200_CHECK_ARG(a->dim >= 1 && a->dim <= kMaxGenericDim, "stream_step: width %d outside 1..%d", a->dim, kMaxGenericDim);
  B200_CHECK_ARG(!a->y || (a->mix && a->out_weight), "stream_step: a result without its mixing weights");
  B200_CHECK_ARG(!a->y2 || (a->y && a->y_norm && a->y2_norm), "stream_step: a second result without norms");
  B200_CHECK_ARG(!a->gate || a->gate_bias, "stream_step: a gate without its bias");
  B200_CHECK_ARG(!a->h || (a->in_weight && a->norm_weight), "stream_step: an input without its weights");
  B200_CHECK_ARG(!a->shifted || (a->h && a->shift && a->previous && a->slots && a->seq_lens && !a->row_ids),
                 "stream_step: a token shift without its state");
  if (a->rows <= 0) return B200_OK;
  return B200_DISPATCH_DTYPE(a->dtype, T, [&]() -> int { return launch_step<T>(*a, (cudaStream_t)stream); });
}

}  // extern "C"
