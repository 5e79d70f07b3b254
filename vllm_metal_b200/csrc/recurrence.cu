// Gated linear recurrences over per-request state slots (include/b200_hybrid_ops.h): Mamba-2, mLSTM and lightning attention share
//   S <- decay S + weight k v^T,   out = S^T q
// and differ in how decay / weight come from the gates (lightning attention has none) and in mLSTM's normaliser.  RWKV-style
// time mixing has a decay per key channel and reads the state before the row's own part, which enters with a weight of its own.
//
//  * sequential form: one CTA per (64-wide value tile, head, segment); the fp32 state is streamed once per token
//    (decode: HBM-bound at 2 * key_dim * value_dim * 4 bytes per head), any type and any size.
//  * chunked forms (bf16 operands), all chunks in parallel: recurrence_tc.cuh (tcgen05, 128 rows) where the key size is
//    whole 64-wide slices, else recurrence_chunk.cuh (warp-level tensor cores, 64 rows); decays per key channel:
//    recurrence_wkv.cuh.
#include "recurrence_tc.cuh"
#include "recurrence_wkv.cuh"

namespace b200 {
namespace rec {

constexpr int kThreads = 256;

template <typename T, int KIND, int VEC>
__global__ void __launch_bounds__(kThreads)
sequential_kernel(const b200_recurrence_args a) {
  extern __shared__ float smem[];
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.z, h = blockIdx.y, tile = blockIdx.x;
  const int row0 = a.cu_seqlens[s], len = a.cu_seqlens[s + 1] - row0;
  if (len <= 0 || len > a.seq_limit) return;
  const int K = a.key_dim, V = a.value_dim, tiles = gridDim.x;
  constexpr int LPR = kTileV / VEC;         // threads across one row of the value tile
  constexpr int RP = kThreads / LPR;        // state rows in flight
  constexpr int BATCH = VEC == 4 ? 8 : 4;   // independent loads per thread
  const int tid = threadIdx.x, col = (tid % LPR) * VEC, row = tid / LPR;
  const int c0 = tile * kTileV;
  const bool live = c0 + col < V;           // VEC = 4 needs V % 4 == 0
  const int g = h / (a.num_heads / a.num_groups);
  float* sq = smem;                         // [K]
  float* sk = sq + K;                       // [K]
  float* sred = sk + K;                     // [RP][64]
  float* sdot = sred + RP * kTileV;         // [8]
  float* sdec = sdot + 8;                   // [K] decays, kind 3
  float* sown = sdec + K;                   // [K] u k, kind 3
  const int64_t slot = a.slots[s];
  float* S = a.state + ((slot * a.num_heads + h) * (int64_t)K) * V + c0 + col;
  float* N = nullptr;
  float* M = nullptr;
  float m = 0.f;
  bool zero = a.seq_lens[s] == len;
  if (KIND == kMlstm) {
    N = a.norm_state + ((slot * a.num_heads + h) * tiles + tile) * (int64_t)K;
    M = a.max_state + (slot * a.num_heads + h) * tiles + tile;
    m = zero ? 0.f : *M;
    __syncthreads();  // every thread has the old maximum before thread 0 replaces it
  }
  for (int t = 0; t < len; ++t) {
    const int64_t r = row0 + t;
    const T* q = reinterpret_cast<const T*>(a.q) + r * a.q_stride + (int64_t)g * K;
    const T* k = reinterpret_cast<const T*>(a.k) + r * a.k_stride + (int64_t)g * K;
    const T* v = reinterpret_cast<const T*>(a.v) + r * a.v_stride + (int64_t)h * V + c0 + col;
    for (int n = tid; n < K; n += kThreads) {
      const float qn = to_float(q[n]), kn = to_float(k[n]);
      sq[n] = (KIND == kLightning && a.silu ? silu_f(qn) : qn) * a.q_scale;
      sk[n] = KIND == kLightning && a.silu ? silu_f(kn) : kn;
      if (KIND == kWkv) {
        const int hn = h * K + n;
        sdec[n] = expf(-expf(reinterpret_cast<const float*>(a.gate_a)[r * a.gate_stride + hn] + a.bias_a[hn]));
        sown[n] = a.skip[hn] * kn;
        sq[n] = qn;
      }
    }
    float vv[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      vv[e] = live ? to_float(v[e]) : 0.f;
      if (KIND == kLightning && a.silu) vv[e] = silu_f(vv[e]);
    }
    const float ga =
        KIND == kLightning || KIND == kWkv ? 0.f : to_float(reinterpret_cast<const T*>(a.gate_a)[r * a.gate_stride + h]);
    float decay, weight;
    if (KIND == kLightning) {
      decay = a.decay[h];
      weight = 1.f;
    } else if (KIND == kWkv) {
      decay = 1.f;  // per key channel, below
      weight = 1.f;
    } else if (KIND == kSsd) {
      const float dt = softplus_f(ga + a.bias_a[h]);
      decay = expf(-a.rate[h] * dt);
      weight = dt;
    } else {
      const float gb = to_float(reinterpret_cast<const T*>(a.gate_b)[r * a.gate_stride + h]);
      const float li = a.gate_cap * tanhf((ga + a.bias_a[h]) / a.gate_cap);
      const float lf = -softplus_f(-a.gate_cap * tanhf((gb + a.bias_b[h]) / a.gate_cap));
      const float mn = fmaxf(lf + m, li);
      decay = expf(lf + m - mn);
      weight = expf(li - mn);
      m = mn;
    }
    __syncthreads();
    float acc[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
    if (live) {
      for (int n0 = row; n0 < K; n0 += RP * BATCH) {
        float st[BATCH][VEC];
#pragma unroll
        for (int j = 0; j < BATCH; ++j) {
          const int n = n0 + j * RP;
          if (n < K && !zero)
            load_vec<VEC>(st[j], S + (int64_t)n * V);
          else
#pragma unroll
            for (int e = 0; e < VEC; ++e) st[j][e] = 0.f;
        }
#pragma unroll
        for (int j = 0; j < BATCH; ++j) {
          const int n = n0 + j * RP;
          if (n < K) {
            const float wk = weight * sk[n], qn = sq[n];
            if (KIND == kWkv) {
              const float d = sdec[n], own = sown[n];
#pragma unroll
              for (int e = 0; e < VEC; ++e) {
                acc[e] += (st[j][e] + own * vv[e]) * qn;
                st[j][e] = d * st[j][e] + wk * vv[e];
              }
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
              if (KIND == kWkv) break;
              st[j][e] = decay * st[j][e] + wk * vv[e];
              acc[e] += st[j][e] * qn;
            }
            store_vec<VEC>(S + (int64_t)n * V, st[j]);
          }
        }
      }
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) sred[row * kTileV + col + e] = acc[e];
    if (KIND == kMlstm) {
      float part = 0.f;
      for (int n = tid; n < K; n += kThreads) {
        const float nn = decay * (zero ? 0.f : N[n]) + weight * sk[n];
        N[n] = nn;
        part += nn * sq[n];
      }
      part = warp_sum(part);
      if ((tid & 31) == 0) sdot[tid >> 5] = part;
    }
    __syncthreads();
    if (tid < kTileV && c0 + tid < V) {
      float y = 0.f;
#pragma unroll
      for (int j = 0; j < RP; ++j) y += sred[j * kTileV + tid];
      if (KIND == kSsd) {
        const T* vr = reinterpret_cast<const T*>(a.v) + r * a.v_stride + (int64_t)h * V + c0;
        y += a.skip[h] * to_float(vr[tid]);
      } else if (KIND == kMlstm) {
        float dot = 0.f;
#pragma unroll
        for (int j = 0; j < kThreads / 32; ++j) dot += sdot[j];
        y /= fmaxf(fabsf(dot), expf(-m)) + 1e-6f;
      }
      reinterpret_cast<T*>(a.out)[r * a.out_stride + (int64_t)h * V + c0 + tid] = from_float<T>(y);
    }
    zero = false;
    __syncthreads();
  }
  if (KIND == kMlstm && tid == 0) *M = m;
}

template <typename T, int KIND>
int launch_sequential(const b200_recurrence_args& a, cudaStream_t st) {
  const int tiles = (a.value_dim + kTileV - 1) / kTileV;
  const bool vec = a.value_dim % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
  const int rp = vec ? kThreads / (kTileV / 4) : kThreads / kTileV;
  const size_t smem = ((KIND == kWkv ? 4 : 2) * (size_t)a.key_dim + (size_t)rp * kTileV + 8) * sizeof(float);
  B200_CHECK_ARG(smem <= 48 * 1024, "recurrence: key_dim %d is too large", a.key_dim);
  const dim3 grid(tiles, a.num_heads, a.num_seqs);
  B200_CUDA_OK(launch_pdl(vec ? sequential_kernel<T, KIND, 4> : sequential_kernel<T, KIND, 1>, grid, dim3(kThreads),
                          smem, st, a));
  return check_launch("recurrence (sequential)");
}

}  // namespace rec
}  // namespace b200

using namespace b200;

namespace {
template <typename T>
int run_sequential(const b200_recurrence_args& a, cudaStream_t st) {
  return a.kind == rec::kSsd     ? rec::launch_sequential<T, rec::kSsd>(a, st)
         : a.kind == rec::kMlstm ? rec::launch_sequential<T, rec::kMlstm>(a, st)
         : a.kind == rec::kWkv   ? rec::launch_sequential<T, rec::kWkv>(a, st)
                                 : rec::launch_sequential<T, rec::kLightning>(a, st);
}
}  // namespace

extern "C" {

size_t b200_recurrence_workspace_bytes(const b200_recurrence_args* a) {
  return a && a->num_chunks > 0 ? rec::Workspace::bytes(*a) : 0;
}

int b200_recurrence_chunk(const b200_recurrence_args* a) {
  if (!a) return 0;
  if (a->kind == rec::kWkv) return rec::can_chunk(*a) ? B200_RECURRENCE_CHUNK : 0;
  return rec::tcr::supported(*a) ? B200_RECURRENCE_CHUNK_TC : rec::can_chunk(*a) ? B200_RECURRENCE_CHUNK : 0;
}

int b200_recurrence_failed(void) {
  int v = 0;
  if (cudaMemcpyFromSymbol(&v, rec::tcr::g_failed, sizeof(v)) != cudaSuccess) return -1;
  return v;
}

int b200_recurrence_num_launches(const b200_recurrence_args* a) {
  return (a->seq_limit > 0 ? 1 : 0) + (a->num_chunks > 0 ? (a->chunk == B200_RECURRENCE_CHUNK_TC ? 4 : 3) : 0);
}

int b200_recurrence(const b200_recurrence_args* a, void* stream) {
  B200_CHECK_ARG(a && a->q && a->k && a->v && a->state && a->out, "recurrence: null argument");
  B200_CHECK_ARG(a->cu_seqlens && a->seq_lens && a->slots, "recurrence: no segments");
  B200_CHECK_ARG(a->kind == rec::kSsd || a->kind == rec::kMlstm || a->kind == rec::kLightning || a->kind == rec::kWkv,
                 "recurrence: unknown kind %d", a->kind);
  B200_CHECK_ARG(a->kind == rec::kLightning || (a->gate_a && a->bias_a), "recurrence: this kind needs its gates");
  B200_CHECK_ARG(!a->silu || (a->kind == rec::kLightning && a->num_chunks <= 0),
                 "recurrence: silu on load is the token-by-token form of kind 2");
  B200_CHECK_ARG(a->num_heads > 0 && a->num_groups > 0 && a->num_heads % a->num_groups == 0,
                 "recurrence: %d heads in %d groups", a->num_heads, a->num_groups);
  B200_CHECK_ARG(a->key_dim > 0 && a->value_dim > 0, "recurrence: empty state");
  if (a->kind == rec::kSsd)
    B200_CHECK_ARG(a->rate && a->skip, "recurrence: kind 0 needs rate and skip");
  else if (a->kind == rec::kWkv)
    B200_CHECK_ARG(a->skip && a->num_groups == a->num_heads, "recurrence: kind 3 needs its bonus and a key per head");
  else if (a->kind == rec::kLightning)
    B200_CHECK_ARG(a->rate && a->decay, "recurrence: kind 2 needs rate and decay");
  else
    B200_CHECK_ARG(a->gate_b && a->bias_b && a->norm_state && a->max_state && a->gate_cap > 0.f,
                   "recurrence: kind 1 needs both gates, its normaliser state and gate_cap > 0");
  if (a->num_seqs <= 0) return B200_OK;
  B200_CHECK_ARG(a->num_seqs <= 65535 && a->num_heads <= 65535, "recurrence: batch too large");
  cudaStream_t st = (cudaStream_t)stream;
  if (a->seq_limit > 0) {
    const int rc = B200_DISPATCH_DTYPE(a->dtype, T, [&]() -> int { return run_sequential<T>(*a, st); });
    if (rc != B200_OK) return rc;
  }
  if (a->num_chunks > 0) {
    if (a->chunk == B200_RECURRENCE_CHUNK_TC) {
      B200_CHECK_ARG(a->kind != rec::kWkv && rec::tcr::supported(*a), "recurrence: this type or these sizes have no tcgen05 form");
      return a->kind == rec::kSsd     ? rec::tcr::launch<rec::kSsd>(*a, st)
             : a->kind == rec::kMlstm ? rec::tcr::launch<rec::kMlstm>(*a, st)
                                      : rec::tcr::launch<rec::kLightning>(*a, st);
    }
    B200_CHECK_ARG(a->chunk == B200_RECURRENCE_CHUNK && rec::can_chunk(*a),
                   "recurrence: this type or these sizes have no chunked form of %d rows", a->chunk);
    if (a->kind == rec::kWkv) return rec::wkv::launch(*a, st);
    return a->kind == rec::kSsd     ? rec::launch_chunked<rec::kSsd>(*a, st)
           : a->kind == rec::kMlstm ? rec::launch_chunked<rec::kMlstm>(*a, st)
                                    : rec::launch_chunked<rec::kLightning>(*a, st);
  }
  return B200_OK;
}

}  // extern "C"
