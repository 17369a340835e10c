// Grouped-head streaming attention, activation format f16.
#include "attn_gqa_impl.cuh"

cudaError_t arcb_attn_gqa_dispatch_f16(const AttnGqaArgs& a, dim3 grid, cudaStream_t stream) {
  return gqa_dispatch<1>(a, grid, stream);
}
