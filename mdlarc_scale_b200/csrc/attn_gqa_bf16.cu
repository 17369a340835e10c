// Grouped-head streaming attention, activation format bf16.
#include "attn_gqa_impl.cuh"

cudaError_t arcb_attn_gqa_dispatch_bf16(const AttnGqaArgs& a, dim3 grid, cudaStream_t stream) {
  return gqa_dispatch<0>(a, grid, stream);
}
