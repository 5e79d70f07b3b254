// The decode kernel's forms that keep 16 significant bits of the softmax weights: bf16, keys and values of any sizes (whole
// 8-element units up to 256).  Four sources instantiate them, PACK and KEEP on and off.
#pragma once

#include "paged_attention_decode.cuh"

namespace b200 {
namespace wide {

template <bool PACK, bool KEEP, int DK, int DV>
int launch(const DecodeParams& p, dim3 grid, cudaStream_t st) {
  return launch_decode_form<__nv_bfloat16, DK, DV, decode_wide_stages(DK, DV), false, true, PACK, KEEP>(p, grid, st);
}

template <bool PACK, bool KEEP, int DK>
int launch(const DecodeParams& p, dim3 grid, cudaStream_t st) {
  switch (decode_value_width(p.value_dim)) {
    case 64: return launch<PACK, KEEP, DK, 64>(p, grid, st);
    case 128: return launch<PACK, KEEP, DK, 128>(p, grid, st);
    case 192: return launch<PACK, KEEP, DK, 192>(p, grid, st);
    default: return launch<PACK, KEEP, DK, 256>(p, grid, st);
  }
}

template <bool PACK, bool KEEP>
int launch(const DecodeParams& p, dim3 grid, cudaStream_t st) {
  switch (decode_key_width(p.head_dim)) {
    case 64: return launch<PACK, KEEP, 64>(p, grid, st);
    case 96: return launch<PACK, KEEP, 96>(p, grid, st);
    case 128: return launch<PACK, KEEP, 128>(p, grid, st);
    default: return launch<PACK, KEEP, 256>(p, grid, st);
  }
}

}  // namespace wide
}  // namespace b200
