// Attention over cached latents on the CUDA cores, for every size and format: the 32-bit path, and what the
// tensor-core kernels are compared with.
//
// One CTA of four warps per (item, head).  A warp takes every fourth key; its lanes share the row, four columns a
// lane and step, and keep the running sums of the same columns.  Scores, weights and sums are fp32; the warps
// merge through shared memory in a fixed order.
#include "attn_latent.cuh"
#include "launch.cuh"

namespace {

constexpr int WARPS = 4;
constexpr float LOG2E = 1.4426950408889634f;

// NV: float4 column steps of 128 that cover kvp
template <int NV>
__global__ void __launch_bounds__(WARPS * 32)
attn_latent_stream_kernel(AttnLatentArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float smem[];          // query [kvp + rotp], then one result of kvp + 4 per warp
  const int lane = threadIdx.x & 31, wj = threadIdx.x >> 5;
  const int item = blockIdx.x / a.n_heads, h = blockIdx.x % a.n_heads;
  const int D = a.kvp + a.rotp;
  float* s_q = smem;
  float* s_part = smem + D;
  const int REC = a.kvp + 4;
  const size_t ih = (size_t)item * a.n_heads + h;
  for (int c = threadIdx.x * 4; c < D; c += WARPS * 128) {
    const float4 v = c < a.kvp ? ld_act4(a.qlat, ih * a.kvp + c, a.fmt)
                               : ld_act4(a.q, ih * a.q_head + a.q_off + (c - a.kvp), a.fmt);
    *reinterpret_cast<float4*>(s_q + c) = v;
  }
  const int seq = a.item_seq ? a.item_seq[item] : item;
  int len = a.item_len[item];
  if (len > a.t_max || seq < 0 || seq >= a.n_seqs) {
    if (threadIdx.x == 0) arcb_set_error(a.err, ARCB_DEV_BAD_INDEX);
    len = 0;
  }
  const int begin = a.window > 0 ? max(0, len - a.window) : 0;
  const float sc = a.scale * LOG2E;
  __syncthreads();

  float m = -INFINITY, l = 0.f;
  float4 acc[NV];
#pragma unroll
  for (int k = 0; k < NV; ++k) acc[k] = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int p = begin + wj; p < len; p += WARPS) {
    const size_t row = ((size_t)seq * (D / 64) * a.t_max + p) * 64;         // of the first panel
    auto at = [&](int c) { return row + (size_t)(c >> 6) * a.t_max * 64 + (c & 63); };
    float4 v[NV];
    float d = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = lane * 4 + k * 128;
      v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < a.kvp) {
        v[k] = ld_act4(a.cache, at(c), a.fmt);
        const float4 q = *reinterpret_cast<const float4*>(s_q + c);
        d += (v[k].x * q.x + v[k].y * q.y) + (v[k].z * q.z + v[k].w * q.w);
      }
    }
    for (int c = a.kvp + lane * 4; c < D; c += 128) {
      const float4 r = ld_act4(a.cache, at(c), a.fmt);
      const float4 q = *reinterpret_cast<const float4*>(s_q + c);
      d += (r.x * q.x + r.y * q.y) + (r.z * q.z + r.w * q.w);
    }
    const float s = warp_sum(d) * sc;
    if (s > m) {
      const float al = exp2f(m - s);
      m = s;
      l *= al;
#pragma unroll
      for (int k = 0; k < NV; ++k) { acc[k].x *= al; acc[k].y *= al; acc[k].z *= al; acc[k].w *= al; }
    }
    const float w = exp2f(s - m);
    l += w;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      acc[k].x += w * v[k].x; acc[k].y += w * v[k].y; acc[k].z += w * v[k].z; acc[k].w += w * v[k].w;
    }
  }
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int c = lane * 4 + k * 128;
    if (c < a.kvp) *reinterpret_cast<float4*>(s_part + wj * REC + c) = acc[k];
  }
  if (lane == 0) {
    s_part[wj * REC + a.kvp] = m;
    s_part[wj * REC + a.kvp + 1] = l;
  }
  __syncthreads();
  const float sk = a.sink ? a.sink[h] * LOG2E : -INFINITY;
  float mt = sk;
#pragma unroll
  for (int j = 0; j < WARPS; ++j) mt = fmaxf(mt, s_part[j * REC + a.kvp]);
  const float ms = mt == -INFINITY ? 0.f : mt;
  float f[WARPS], lt = exp2f(sk - ms);
#pragma unroll
  for (int j = 0; j < WARPS; ++j) {
    f[j] = exp2f(s_part[j * REC + a.kvp] - ms);
    lt += s_part[j * REC + a.kvp + 1] * f[j];
  }
  const float inv = lt > 0.f ? 1.f / lt : 0.f;
  for (int c = threadIdx.x; c < a.kvp; c += WARPS * 32) {
    float o = 0.f;
#pragma unroll
    for (int j = 0; j < WARPS; ++j) o += s_part[j * REC + c] * f[j];
    st_act(a.out, ih * a.kvp + c, o * inv, a.fmt);
  }
}

template <int NV>
cudaError_t launch(const AttnLatentArgs& a, cudaStream_t stream) {
  const size_t smem = ((size_t)a.kvp + a.rotp + WARPS * (a.kvp + 4)) * 4;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(attn_latent_stream_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return arcb_launch(attn_latent_stream_kernel<NV>, dim3((unsigned)(a.n_items * a.n_heads)), dim3(WARPS * 32), smem, stream, a);
}

}  // namespace

int arcb_launch_attn_latent_stream(const AttnLatentArgs& a, cudaStream_t stream) {
  if (a.n_items <= 0) return 0;
  if (a.kvp % 64 || a.rotp % 64 || a.q_head % 4 || a.q_off % 4 || (long long)a.n_items * a.n_heads > 0x7fffffffLL) return -1;
  cudaError_t e;
  if (a.kvp <= 128) e = launch<1>(a, stream);
  else if (a.kvp <= 256) e = launch<2>(a, stream);
  else if (a.kvp <= 512) e = launch<4>(a, stream);
  else if (a.kvp <= 1024) e = launch<8>(a, stream);
  else if (a.kvp <= 2048) e = launch<16>(a, stream);
  else return -1;
  arcb_count_launch(1);
  return (int)e;
}
