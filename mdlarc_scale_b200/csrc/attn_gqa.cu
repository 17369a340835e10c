// Launcher of the grouped-head streaming attention (one query row per item) and the merge of its splits.
#include "attn_gqa.cuh"
#include "launch.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

// One warp per (item, head): merges the splits in order, adds the sink, applies the gate.
__global__ void __launch_bounds__(128)
attn_gqa_combine_kernel(AttnGqaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long ih = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (ih >= (long long)a.n_items * a.n_heads) return;
  const int item = (int)(ih / a.n_heads), h = (int)(ih % a.n_heads);
  const int rec = a.vdimp + 4;
  const float* r0 = a.scratch + (size_t)ih * a.n_splits * rec;
  const float sk = a.sink ? a.sink[h] * LOG2E : -INFINITY;
  float m = sk;
  for (int s = 0; s < a.n_splits; ++s) m = fmaxf(m, r0[(size_t)s * rec + a.vdimp]);
  const float ms = (m == -INFINITY) ? 0.f : m;
  float l = exp2f(sk - ms);
  for (int s = 0; s < a.n_splits; ++s) l += r0[(size_t)s * rec + a.vdimp + 1] * exp2f(r0[(size_t)s * rec + a.vdimp] - ms);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int c = lane; c < a.vdimp; c += 32) {
    float o = 0.f;
    for (int s = 0; s < a.n_splits; ++s) o += r0[(size_t)s * rec + c] * exp2f(r0[(size_t)s * rec + a.vdimp] - ms);
    o *= inv;
    if (a.gate) o *= ld_act(a.gate, (size_t)item * a.gate_pitch + (size_t)h * a.vdimp + c, a.fmt);
    st_act(a.out, (size_t)ih * a.vdimp + c, o, a.fmt);
  }
}

int tiles_of(int rep) { return (rep + 3) / 4; }

}  // namespace

int arcb_attn_gqa_splits(int n_items, int n_kv, int rep, int t_max) {
  // four-warp CTAs: at least three for each of the 148 SMs, with at least 128 cached rows per split
  const long long work = (long long)n_items * n_kv * tiles_of(rep);
  long long s = (148LL * 3 + work - 1) / work;
  if (t_max > 0 && s > t_max / 128) s = t_max / 128;
  if (s < 1) s = 1;
  if (s > 32) s = 32;
  return (int)s;
}

int arcb_launch_attn_gqa(AttnGqaArgs a, cudaStream_t stream) {
  if (a.n_items <= 0) return 0;
  if (a.n_kv <= 0 || a.n_heads % a.n_kv || a.n_splits < 1 || (a.n_splits > 1 && !a.scratch)) return -1;
  a.rep = a.n_heads / a.n_kv;
  a.tiles = tiles_of(a.rep);
  a.tile_rows = (a.rep + a.tiles - 1) / a.tiles;
  const long long blocks = (long long)a.n_items * a.n_kv * a.tiles * a.n_splits;
  if (blocks > 0x7fffffffLL) return -1;
  const dim3 grid((unsigned)blocks);
  cudaError_t e = a.fmt == 2 ? arcb_attn_gqa_dispatch_f32(a, grid, stream)
                : a.fmt == 1 ? arcb_attn_gqa_dispatch_f16(a, grid, stream)
                             : arcb_attn_gqa_dispatch_bf16(a, grid, stream);
  arcb_count_launch(1);
  if (e == cudaSuccess && a.n_splits > 1) return arcb_launch_attn_combine(a, stream);
  return (int)e;
}

int arcb_launch_attn_combine(const AttnGqaArgs& a, cudaStream_t stream) {
  const long long nb = ((long long)a.n_items * a.n_heads + 3) / 4;
  const cudaError_t e = arcb_launch(attn_gqa_combine_kernel, dim3((unsigned)nb), dim3(128), 0, stream, a);
  arcb_count_launch(1);
  return (int)e;
}
