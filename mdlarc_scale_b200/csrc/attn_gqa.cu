// Launcher of the grouped-head streaming attention (one query row per item) and the merge of its splits.
#include "attn_gqa.cuh"
#include "launch.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

// One warp per (item, head): merges the splits in order, adds the sink, applies the gate.  Lane s keeps the factor of
// splits s and s + 32.
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
  float m_s[2], l_s[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int s = lane + 32 * i;
    const float2 ml = s < a.n_splits ? *reinterpret_cast<const float2*>(r0 + (size_t)s * rec + a.vdimp) : make_float2(-INFINITY, 0.f);
    m_s[i] = ml.x;
    l_s[i] = ml.y;
  }
  const float sk = a.sink ? a.sink[h] * LOG2E : -INFINITY;
  float m = fmaxf(m_s[0], m_s[1]);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
  m = fmaxf(m, sk);
  const float ms = (m == -INFINITY) ? 0.f : m;
  const float f0 = exp2f(m_s[0] - ms), f1 = exp2f(m_s[1] - ms);
  const float l = warp_sum(l_s[0] * f0 + l_s[1] * f1) + exp2f(sk - ms);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int c = lane * 4; c < ((a.vdimp + 127) & ~127); c += 128) {       // every lane takes every step: the shuffles need them
    const bool in = c < a.vdimp;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < a.n_splits; ++s) {
      const float f = __shfl_sync(0xffffffffu, s < 32 ? f0 : f1, s & 31);
      if (in) {
        const float4 v = *reinterpret_cast<const float4*>(r0 + (size_t)s * rec + c);
        o.x += v.x * f; o.y += v.y * f; o.z += v.z * f; o.w += v.w * f;
      }
    }
    if (!in) continue;
    o.x *= inv; o.y *= inv; o.z *= inv; o.w *= inv;
    if (a.gate) {
      const float4 g = ld_act4(a.gate, (size_t)item * a.gate_pitch + (size_t)h * a.vdimp + c, a.fmt);
      o.x *= g.x; o.y *= g.y; o.z *= g.z; o.w *= g.w;
    }
    st_act4(a.out, (size_t)ih * a.vdimp + c, o, a.fmt);
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
