#include "paged_attention_decode_wide.cuh"

namespace b200 {

int launch_decode_wide(const DecodeParams& p, dim3 grid, cudaStream_t st) { return wide::launch<false, false>(p, grid, st); }

}  // namespace b200
