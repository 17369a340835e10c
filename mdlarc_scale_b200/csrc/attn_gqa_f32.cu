// Grouped-head streaming attention, activation format f32.
#include "attn_gqa_impl.cuh"

cudaError_t arcb_attn_gqa_dispatch_f32(const AttnGqaArgs& a, dim3 grid, cudaStream_t stream) {
  return gqa_dispatch<2>(a, grid, stream);
}
