#include "paged_attention_decode_wide.cuh"

namespace b200 {

int launch_decode_kept(const DecodeParams& p, dim3 grid, cudaStream_t st) { return wide::launch<false, true>(p, grid, st); }

}  // namespace b200
