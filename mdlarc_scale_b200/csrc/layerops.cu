// Row-wise kernels of layered models:
//   lm_embed / step_begin : embedding -> residual stream (+ the decode step's positions)
//   lm_norm               : norm of the residual stream -> GEMM operand, and the scaled residual in place
//   sandwich_norm         : norm of a sublayer's output, residual sum and the next sublayer's norm in one pass
//   latent_prep           : query latent, cached latent and rotated key part from their fp32 projections
//   proj_prep             : head norms, query gain, gates and cache writes of a projection left in fp32
//   pick                  : logit scale, argmax or temperature / top-k sampling, decode bookkeeping
// Norms, gates, angles and the residual are fp32 throughout; fmt selects the operand format.
#include "../../include/arcb200.h"
#include "layerops.cuh"
#include "launch.cuh"

namespace {

constexpr int ROWS_PER_CTA = 4;

__device__ __forceinline__ void embed_row(const LmEmbedArgs& a, int row, int tok, int lane) {
  tok = min(max(tok, 0), a.vocab - 1);
  const float* src = a.embed + (size_t)tok * a.pitch;
  float* x = a.x + (size_t)row * a.pitch;
  for (int i = lane * 4; i < a.pitch; i += 128) {   // the table's padding columns are zero
    const float4 v = __ldg(reinterpret_cast<const float4*>(src + i));
    if (a.xn) st_act4(a.xn, (size_t)row * a.pitch + i, v, a.fmt);
    *reinterpret_cast<float4*>(x + i) = make_float4(a.alpha * v.x, a.alpha * v.y, a.alpha * v.z, a.alpha * v.w);
  }
}

__device__ __forceinline__ void embed_zero(const LmEmbedArgs& a) {
  if (blockIdx.x == 0)
    for (int i = threadIdx.x; i < a.n_zero; i += blockDim.x) a.zero[i] = 0;
}

__global__ void __launch_bounds__(ROWS_PER_CTA * 32)
lm_embed_kernel(LmEmbedArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  embed_zero(a);
  const int row = blockIdx.x * ROWS_PER_CTA + (threadIdx.x >> 5);
  if (row >= a.rows) return;
  embed_row(a, row, a.token_ids[row], threadIdx.x & 31);
}

__global__ void __launch_bounds__(ROWS_PER_CTA * 32)
step_begin_kernel(StepState st, LmEmbedArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  embed_zero(a);
  const int b = blockIdx.x * ROWS_PER_CTA + (threadIdx.x >> 5);
  if (b >= st.n_seqs) return;
  const int lane = threadIdx.x & 31;
  if (lane == 0) {
    int pos = st.active[b] ? st.cur_len[b] : -1;
    if (pos >= st.t_max) {          // the cache row is full: hold the sequence
      arcb_set_error(st.err, ARCB_DEV_BAD_INDEX);
      st.active[b] = 0;
      pos = -1;
    }
    st.pos[b] = pos;
    st.kv_len[b] = pos + 1;
  }
  embed_row(a, b, st.cur_tok[b], lane);
}

// One warp per row.  Rows of up to 128 * NV floats stay in registers: one read of the row, and the
// deviations are formed from the registers (two-pass variance).
template <int NV>
__device__ __forceinline__ void norm_row_regs(const LmNormArgs& a, float* __restrict__ x, int row, int lane) {
  float4 v[NV];
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = lane * 4 + k * 128;
    v[k] = (i < a.pitch) ? *reinterpret_cast<const float4*>(x + i) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const float inv_n = 1.f / (float)a.width;
  float mean = 0.f;
  if (a.kind == ARCB_NORM_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) s += (v[k].x + v[k].y) + (v[k].z + v[k].w);   // padding columns are zero
    mean = warp_sum(s) * inv_n;
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = lane * 4 + k * 128;
    v[k].x = i < a.width ? v[k].x - mean : 0.f;
    v[k].y = i + 1 < a.width ? v[k].y - mean : 0.f;
    v[k].z = i + 2 < a.width ? v[k].z - mean : 0.f;
    v[k].w = i + 3 < a.width ? v[k].w - mean : 0.f;
    ss += (v[k].x * v[k].x + v[k].y * v[k].y) + (v[k].z * v[k].z + v[k].w * v[k].w);
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) * inv_n + a.eps);
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = lane * 4 + k * 128;
    if (i < a.pitch) {
      const float4 g = __ldg(reinterpret_cast<const float4*>(a.w + i));
      const float4 y = make_float4((v[k].x * inv) * g.x, (v[k].y * inv) * g.y, (v[k].z * inv) * g.z, (v[k].w * inv) * g.w);
      st_act4(a.xn, (size_t)row * a.pitch + i, y, a.fmt);
      if (a.write_x)
        *reinterpret_cast<float4*>(x + i) = make_float4(a.x_scale * y.x, a.x_scale * y.y, a.x_scale * y.z, a.x_scale * y.w);
      if (a.dense) {
        float* dp = a.dense + (size_t)row * a.width;
        if (i < a.width) dp[i] = y.x;
        if (i + 1 < a.width) dp[i + 1] = y.y;
        if (i + 2 < a.width) dp[i + 2] = y.z;
        if (i + 3 < a.width) dp[i + 3] = y.w;
      }
    }
  }
}

// Wide rows: three passes over the row in memory (L1/L2-resident after the first).
__device__ __forceinline__ void norm_row_loop(const LmNormArgs& a, float* __restrict__ x, int row, int lane) {
  const float inv_n = 1.f / (float)a.width;
  float mean = 0.f;
  if (a.kind == ARCB_NORM_LAYER) {
    float s = 0.f;
    for (int i = lane * 4; i < a.pitch; i += 128) {
      const float4 v = *reinterpret_cast<const float4*>(x + i);
      s += (v.x + v.y) + (v.z + v.w);
    }
    mean = warp_sum(s) * inv_n;
  }
  float ss = 0.f;
  for (int i = lane; i < a.width; i += 32) {
    const float d = x[i] - mean;
    ss += d * d;
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) * inv_n + a.eps);
  for (int i = lane * 4; i < a.pitch; i += 128) {
    const float4 v = *reinterpret_cast<const float4*>(x + i);
    const float4 g = __ldg(reinterpret_cast<const float4*>(a.w + i));   // gains of padding columns are zero
    const float4 y = make_float4(((v.x - mean) * inv) * g.x, ((v.y - mean) * inv) * g.y, ((v.z - mean) * inv) * g.z,
                                 ((v.w - mean) * inv) * g.w);
    st_act4(a.xn, (size_t)row * a.pitch + i, y, a.fmt);
    if (a.write_x)
      *reinterpret_cast<float4*>(x + i) = make_float4(a.x_scale * y.x, a.x_scale * y.y, a.x_scale * y.z, a.x_scale * y.w);
    if (a.dense) {
      const float yv[4] = {y.x, y.y, y.z, y.w};
      for (int j = 0; j < 4; ++j)
        if (i + j < a.width) a.dense[(size_t)row * a.width + i + j] = yv[j];
    }
  }
}

__global__ void __launch_bounds__(ROWS_PER_CTA * 32)
lm_norm_kernel(LmNormArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x * ROWS_PER_CTA + (threadIdx.x >> 5);
  if (row >= a.rows) return;
  const int lane = threadIdx.x & 31;
  float* x = a.x + (size_t)(a.row_index ? a.row_index[row] : row) * a.pitch;
  if (a.pitch <= 128 * 2) norm_row_regs<2>(a, x, row, lane);
  else if (a.pitch <= 128 * 6) norm_row_regs<6>(a, x, row, lane);
  else if (a.pitch <= 128 * 10) norm_row_regs<10>(a, x, row, lane);
  else if (a.pitch <= 128 * 16) norm_row_regs<16>(a, x, row, lane);
  else norm_row_loop(a, x, row, lane);
}

// Sum over a CTA of WARPS warps; every thread gets it.  Two calls in a row need different `sm`.
template <int WARPS>
__device__ __forceinline__ float cta_sum(float v, float* sm) {
  v = warp_sum(v);
  if constexpr (WARPS == 1) return v;
  if ((threadIdx.x & 31) == 0) sm[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = sm[0];
#pragma unroll
  for (int i = 1; i < WARPS; ++i) t += sm[i];
  return t;
}

__device__ __forceinline__ float sum_sq(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }

// One CTA of four warps per row; NV float4 per thread hold the row (REGS) or every pass reads it again.  AHEAD: the
// residual row is loaded beside the sublayer's output (few rows: shorter; many rows: the registers are worth more).
template <int NV, bool REGS, bool AHEAD>
__global__ void __launch_bounds__(128)
sandwich_norm_kernel(SandwichArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sm[2][4];
  const int row = blockIdx.x, tid = threadIdx.x;
  float* x = a.x + (size_t)row * a.pitch;
  const float* y = a.y ? a.y + (size_t)row * a.pitch : nullptr;
  const float inv_n = 1.f / (float)a.width;
  auto sublayer = [&](int i) {
    float4 v = y ? *reinterpret_cast<const float4*>(y + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    if (a.ye)
      for (int k = 0; k < a.top; ++k) {
        const float4 e = ld_act4(a.ye, (size_t)a.slot[(size_t)row * a.top + k] * a.pitch + i, a.fmt);
        v.x += e.x; v.y += e.y; v.z += e.z; v.w += e.w;
      }
    return v;
  };
  auto added = [&](int i, float4 r, float4 v, float inv) {
    const float4 g = __ldg(reinterpret_cast<const float4*>(a.w_out + i));
    return make_float4(r.x + (v.x * inv) * g.x, r.y + (v.y * inv) * g.y, r.z + (v.z * inv) * g.z, r.w + (v.w * inv) * g.w);
  };
  auto dense = [&](int i, float4 v) {
    float* d = a.dense + (size_t)row * a.width;
    if (i < a.width) d[i] = v.x;
    if (i + 1 < a.width) d[i + 1] = v.y;
    if (i + 2 < a.width) d[i + 2] = v.z;
    if (i + 3 < a.width) d[i + 3] = v.w;
  };
  const float* emb = a.embed ? a.embed + (size_t)min(max(a.tokens[row], 0), a.vocab - 1) * a.pitch : nullptr;
  auto with_embed = [&](int i, float4 v) {
    if (emb) {
      const float4 e = __ldg(reinterpret_cast<const float4*>(emb + i));
      v.x += e.x; v.y += e.y; v.z += e.z; v.w += e.w;
    }
    return v;
  };
  auto write_xn = [&](int i, float4 v, float inv) {
    const float4 g = __ldg(reinterpret_cast<const float4*>(a.w_in + i));
    st_act4(a.xn, (size_t)row * a.pitch + i, make_float4((v.x * inv) * g.x, (v.y * inv) * g.y, (v.z * inv) * g.z, (v.w * inv) * g.w), a.fmt);
  };
  // padding columns are zero in y, x, the embedding and the gains
  if constexpr (REGS) {
    float4 v[NV], r[AHEAD ? NV : 1];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (tid + k * 128) * 4;
      v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (i < a.pitch) {
        if constexpr (AHEAD) r[k] = *reinterpret_cast<const float4*>(x + i);
        v[k] = sublayer(i);
      }
      ss += sum_sq(v[k]);
    }
    float inv = 1.f / sqrtf(cta_sum<4>(ss, sm[0]) * inv_n + a.eps);
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (tid + k * 128) * 4;
      if (i >= a.pitch) continue;
      v[k] = added(i, AHEAD ? r[AHEAD ? k : 0] : *reinterpret_cast<const float4*>(x + i), v[k], inv);
      if (a.dense) dense(i, v[k]);
      v[k] = with_embed(i, v[k]);
      *reinterpret_cast<float4*>(x + i) = v[k];
      ss += sum_sq(v[k]);
    }
    if (!a.w_in) return;
    inv = 1.f / sqrtf(cta_sum<4>(ss, sm[1]) * inv_n + a.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (tid + k * 128) * 4;
      if (i < a.pitch) write_xn(i, v[k], inv);
    }
  } else {
    float ss = 0.f;
    for (int i = tid * 4; i < a.pitch; i += 512) ss += sum_sq(sublayer(i));
    float inv = 1.f / sqrtf(cta_sum<4>(ss, sm[0]) * inv_n + a.eps);
    ss = 0.f;
    for (int i = tid * 4; i < a.pitch; i += 512) {
      float4 v = added(i, *reinterpret_cast<const float4*>(x + i), sublayer(i), inv);
      if (a.dense) dense(i, v);
      v = with_embed(i, v);
      *reinterpret_cast<float4*>(x + i) = v;
      ss += sum_sq(v);
    }
    if (!a.w_in) return;
    inv = 1.f / sqrtf(cta_sum<4>(ss, sm[1]) * inv_n + a.eps);
    for (int i = tid * 4; i < a.pitch; i += 512) write_xn(i, *reinterpret_cast<const float4*>(x + i), inv);
  }
}

// One CTA of four warps per row; NV float4 per thread hold the whole row of projections, both norms' sums are taken in
// one exchange.
template <int NV>
__global__ void __launch_bounds__(128)
latent_prep_kernel(LatentPrepArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float2 sm[4];
  const int row = blockIdx.x, tid = threadIdx.x;
  const int pos = a.pos[row], seq = a.seq ? a.seq[row] : row;
  const float* p = a.proj + (size_t)row * a.pitch;
  const int width = a.off_r + a.rotp;
  float4 v[NV];
  float sq = 0.f, sc = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int c = (tid + k * 128) * 4;
    v[k] = c < width ? *reinterpret_cast<const float4*>(p + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int c = (tid + k * 128) * 4;
    if (c < a.off_c) sq += sum_sq(v[k]);
    else if (c < a.off_r) sc += sum_sq(v[k]);
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if ((tid & 31) == 0) sm[tid >> 5] = make_float2(sq, sc);
  __syncthreads();
  sq = (sm[0].x + sm[1].x) + (sm[2].x + sm[3].x);
  sc = (sm[0].y + sm[1].y) + (sm[2].y + sm[3].y);
  const float iq = 1.f / sqrtf(sq / (float)a.q_rank + a.eps), ic = 1.f / sqrtf(sc / (float)a.kv_rank + a.eps);
  const bool bad = pos >= a.t_max || seq < 0 || seq >= a.n_seqs;
  if (bad && pos >= 0 && tid == 0) arcb_set_error(a.err, ARCB_DEV_BAD_INDEX);
  const bool store = pos >= 0 && !bad;
  const size_t row0 = ((size_t)seq * ((a.kv_rankp + a.rotp) >> 6) * a.t_max + pos) * 64, panel = (size_t)a.t_max * 64;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int c = (tid + k * 128) * 4;
    if (c < a.off_c) {
      const float4 g = __ldg(reinterpret_cast<const float4*>(a.q_norm + c));
      st_act4(a.cq, (size_t)row * a.q_rankp + c,
              make_float4((v[k].x * iq) * g.x, (v[k].y * iq) * g.y, (v[k].z * iq) * g.z, (v[k].w * iq) * g.w), a.fmt);
    } else if (c < width && store) {
      float4 o = v[k];
      if (c < a.off_r) {
        const float4 g = __ldg(reinterpret_cast<const float4*>(a.kv_norm + c - a.off_c));
        o = make_float4((o.x * ic) * g.x, (o.y * ic) * g.y, (o.z * ic) * g.z, (o.w * ic) * g.w);
      } else if (a.rot) {
        o = rotate4(o, __ldg(reinterpret_cast<const float4*>(a.rot + (size_t)pos * (a.rotp >> 1) + ((c - a.off_r) >> 1))));
      }
      const int cc = c - a.off_c;
      st_act4(a.cache, row0 + (size_t)(cc >> 6) * panel + (cc & 63), o, a.fmt);
    }
  }
}

// Angles in double precision: a position times a frequency loses nothing before the sine.
__global__ void rot_table_kernel(float2* table, int t_max, int pairs, int dims, double base) {
  const long long n = (long long)t_max * pairs;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const int p = (int)(i / pairs), k = (int)(i - (long long)p * pairs);
    double s = 0., c = 1.;
    if (2 * k < dims) sincos(p * pow(base, -2.0 * k / dims), &s, &c);
    table[i] = make_float2((float)c, (float)s);
  }
}

// One warp per (row, head of a section): 4 consecutive columns per lane and 128-column step.
__global__ void __launch_bounds__(128)
proj_prep_kernel(ProjArgs a, const float* __restrict__ proj, int n_units) {
  pdl_launch_dependents();
  pdl_wait();
  const long long w = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (w >= (long long)a.M * n_units) return;
  const int lane = threadIdx.x & 31;
  const int m = (int)(w / n_units);
  int u = (int)(w - (long long)m * n_units);
  const float* row = proj + (size_t)m * a.N;
  const int nkv = a.recurrent ? a.H : a.G;
  enum { Q, K, V, GATE, LOGS } sec;
  int h;
  if (u < a.H) { sec = Q; h = u; }
  else if ((u -= a.H) < a.H) { sec = GATE; h = u; }
  else if (u -= a.H, a.off_k >= 0 && u < nkv) { sec = K; h = u; }
  else if (a.off_k >= 0 && u < 2 * nkv) { sec = V; h = u - nkv; }
  else { sec = LOGS; h = 0; }

  if (sec == LOGS) {      // recurrence only: the gates of all heads
    for (int j = lane; j < 2 * a.H; j += 32) {
      const int c = a.off_gate + j;
      a.gates[(size_t)m * 2 * a.H + j] = row[c] + (a.bias ? a.bias[c] : 0.f);
    }
    return;
  }
  if (sec == GATE && a.off_g < 0) return;
  const int width = (sec == Q || sec == K) ? a.dimp : a.vdimp;
  const int off = (sec == Q ? a.off_q : sec == K ? a.off_k : sec == V ? a.off_v : a.off_g) + h * width;
  const float* gain = sec == Q ? a.q_norm : sec == K ? a.k_norm : nullptr;
  float4 v[2];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int c = lane * 4 + k * 128;
    v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < width) {
      v[k] = *reinterpret_cast<const float4*>(row + off + c);
      if (a.bias) {
        const float4 b = __ldg(reinterpret_cast<const float4*>(a.bias + off + c));
        v[k].x += b.x; v[k].y += b.y; v[k].z += b.z; v[k].w += b.w;
      }
      ss += (v[k].x * v[k].x + v[k].y * v[k].y) + (v[k].z * v[k].z + v[k].w * v[k].w);
    }
  }
  if (gain) {
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)a.dim + a.eps);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int c = lane * 4 + k * 128;
      if (c < width) {
        const float4 g = __ldg(reinterpret_cast<const float4*>(gain + c));
        v[k] = make_float4((v[k].x * inv) * g.x, (v[k].y * inv) * g.y, (v[k].z * inv) * g.z, (v[k].w * inv) * g.w);
      }
    }
  }
  if (sec == Q) {
    const float f = query_gain(a, a.pos ? max(a.pos[m], 0) : 0);
#pragma unroll
    for (int k = 0; k < 2; ++k) { v[k].x *= f; v[k].y *= f; v[k].z *= f; v[k].w *= f; }
  }
  if (sec == GATE) {
#pragma unroll
    for (int k = 0; k < 2; ++k)
      v[k] = make_float4(sigmoid_exact(v[k].x), sigmoid_exact(v[k].y), sigmoid_exact(v[k].z), sigmoid_exact(v[k].w));
  }
  void* dst = a.out;
  size_t at = (size_t)m * a.N + off;
  if (!a.recurrent && (sec == K || sec == V)) {
    const long long cr = proj_cache_row(a, m);
    if (cr < 0) return;
    dst = sec == K ? a.kcache : a.vcache;
    at = (size_t)(cr + (long long)h * a.t_max) * width;
  }
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int c = lane * 4 + k * 128;
    if (c < width) st_act4(dst, at + c, v[k], a.fmt);
  }
}

// ---- token picking: one CTA per row ----
constexpr int PICK_THREADS = 512;

// Order-preserving map of a float to an unsigned key.
__device__ __forceinline__ uint32_t float_key(float f) {
  const uint32_t b = __float_as_uint(f);
  return (b & 0x80000000u) ? ~b : (b | 0x80000000u);
}

template <typename T, typename Op>
__device__ __forceinline__ T block_reduce(T v, Op op, T* sm) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = op(v, __shfl_xor_sync(0xffffffffu, v, o));
  __syncthreads();
  if ((threadIdx.x & 31) == 0) sm[threadIdx.x >> 5] = v;
  __syncthreads();
  T r = sm[0];
#pragma unroll
  for (int i = 1; i < PICK_THREADS / 32; ++i) r = op(r, sm[i]);
  return r;
}

// Exclusive prefix sum over the CTA's threads.
template <typename T>
__device__ __forceinline__ T block_exclusive(T v, T* sm) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  T inc = v;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const T t = __shfl_up_sync(0xffffffffu, inc, o);
    if (lane >= o) inc += t;
  }
  __syncthreads();
  if (lane == 31) sm[warp] = inc;
  __syncthreads();
  T base = 0;
  for (int i = 0; i < warp; ++i) base += sm[i];
  return base + inc - v;
}

__global__ void __launch_bounds__(PICK_THREADS)
pick_kernel(PickArgs a, StepState st) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float smf[PICK_THREADS / 32];
  __shared__ unsigned long long sml[PICK_THREADS / 32];
  __shared__ int smi[PICK_THREADS / 32];
  __shared__ int s_pick;
  const int i = blockIdx.x, tid = threadIdx.x;
  float* lg = a.logits + (size_t)i * a.pitch;
  int b = -1;
  bool held = false;
  if (a.mode == PICK_FIRST) b = a.first_seq[i];
  else if (a.mode == PICK_DECODE) { b = i; held = !st.active[b]; }
  const bool bad = a.mode != PICK_PLAIN && (b < 0 || b >= st.n_seqs);
  int out_idx = -1;
  if (!bad && a.mode == PICK_FIRST) out_idx = 0;
  else if (!bad && a.mode == PICK_DECODE) out_idx = st.cur_len[b] - st.len0[b] + 1;
  const bool in_range = out_idx >= 0 && out_idx < st.max_new;

  // scale, copy out, first maximum
  unsigned long long best = 0;
  float* step = (!bad && !held && in_range && st.step_logits) ? st.step_logits + ((size_t)b * st.max_new + out_idx) * a.vocab : nullptr;
  for (int v0 = tid * 4; v0 < a.vocab; v0 += PICK_THREADS * 4) {     // rows are padded to a multiple of 128
    float4 f = *reinterpret_cast<const float4*>(lg + v0);
    f.x *= a.scale; f.y *= a.scale; f.z *= a.scale; f.w *= a.scale;
    *reinterpret_cast<float4*>(lg + v0) = f;
    const float xs[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int v = v0 + e;
      if (v >= a.vocab) break;
      if (a.out) a.out[(size_t)i * a.vocab + v] = xs[e];
      if (step) step[v] = xs[e];
      const unsigned long long key = ((unsigned long long)float_key(xs[e]) << 32) | (uint32_t)~v;
      best = key > best ? key : best;
    }
  }
  if (a.mode == PICK_PLAIN || held) return;
  if (bad) { if (tid == 0) arcb_set_error(st.err, ARCB_DEV_BAD_INDEX); return; }
  best = block_reduce(best, [](unsigned long long p, unsigned long long q) { return p > q ? p : q; }, sml);
  int pick = (int)~(uint32_t)best;

  if (st.temperature > 0.f) {
    __syncthreads();
    const float top = lg[pick];
    const float inv_t = 1.f / fmaxf(st.temperature, 1e-6f);
    const int kk = (st.top_k > 0 && st.top_k < a.vocab) ? st.top_k : a.vocab;
    // key of the kk-th largest logit, by bisection over the 32-bit keys
    uint32_t thr = 0;
    if (kk < a.vocab) {
      for (int bit = 31; bit >= 0; --bit) {
        const uint32_t cand = thr | (1u << bit);
        int n = 0;
        for (int v = tid; v < a.vocab; v += PICK_THREADS) n += float_key(lg[v]) >= cand ? 1 : 0;
        n = block_reduce(n, [](int p, int q) { return p + q; }, smi);
        if (n >= kk) thr = cand;
      }
    }
    // contiguous ranges per thread keep index order; of the logits equal to the threshold the first ones stay
    const int per = (a.vocab + PICK_THREADS - 1) / PICK_THREADS;
    const int v0 = min(tid * per, a.vocab), v1 = min(v0 + per, a.vocab);
    int above = 0, equal = 0;
    for (int v = v0; v < v1; ++v) {
      const uint32_t key = float_key(lg[v]);
      above += key > thr ? 1 : 0;
      equal += key == thr ? 1 : 0;
    }
    const int n_above = block_reduce(above, [](int p, int q) { return p + q; }, smi);
    const int eq_before = block_exclusive(equal, smi);
    const int eq_keep = kk - n_above;
    auto weight = [&](int v, int& eq) -> float {
      const float x = lg[v];
      const uint32_t key = float_key(x);
      bool keep = key > thr;
      if (key == thr) keep = eq++ < eq_keep;
      return keep ? __expf((x - top) * inv_t) : 0.f;
    };
    float mine = 0.f;
    int eq = eq_before;
    for (int v = v0; v < v1; ++v) mine += weight(v, eq);
    const float before = block_exclusive(mine, smf);
    __shared__ float s_total;
    if (tid == PICK_THREADS - 1) s_total = before + mine;
    if (tid == 0) s_pick = pick;
    __syncthreads();
    const unsigned long long sid = st.sample_stream ? (unsigned long long)(unsigned int)st.sample_stream[b] : (unsigned long long)b;
    unsigned long long z = st.sample_seed + 0x9E3779B97F4A7C15ull * (sid + 1) + 0xD1B54A32D192ED03ull * (unsigned long long)(out_idx + 1);
    z = (z ^ (z >> 30)) * 0xBF58476D1CE4E5B9ull;
    z = (z ^ (z >> 27)) * 0x94D049BB133111EBull;
    z ^= z >> 31;
    const float u = (float)(z >> 40) * (1.f / 16777216.f) * s_total;
    if (u >= before && u < before + mine) {     // at most one thread: the ranges are disjoint
      float run = before;
      eq = eq_before;
      for (int v = v0; v < v1; ++v) {
        const float p = weight(v, eq);
        run += p;
        if (p > 0.f) { s_pick = v; if (u < run) break; }
      }
    }
    __syncthreads();
    pick = s_pick;
  }
  if (tid != 0) return;
  if (a.mode == PICK_FIRST) {
    st.len0[b] = a.prompt_len[i];
    st.cur_len[b] = a.prompt_len[i];
    st.active[b] = 1;
    if (st.finished[b]) { st.finished[b] = 0; atomicSub(st.n_finished, 1); }
  } else {
    st.cur_len[b] = min(st.cur_len[b] + 1, st.t_max);
  }
  int tok = pick;
  if (in_range) {
    if (st.forced) tok = st.forced[(size_t)b * st.max_new + out_idx];
    st.out_tokens[(size_t)b * st.max_new + out_idx] = tok;
  }
  const bool ended = st.stop_on_end && st.end_token >= 0 && tok == st.end_token;
  const bool spent = out_idx + 1 >= st.max_new;
  if (ended || spent) {
    if (!st.finished[b]) {
      st.finished[b] = 1;
      atomicAdd(st.n_finished, 1);
    }
    if (spent || st.stop_on_end == 1) st.active[b] = 0;
  }
  st.cur_tok[b] = tok;
}

__global__ void seg_commit_kernel(StepState st, const int* seg_seq, const int* seg_pos0, const int* seg_rows, int n) {
  pdl_launch_dependents();
  pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int b = seg_seq[i];
  if (b < 0 || b >= st.n_seqs) { arcb_set_error(st.err, ARCB_DEV_BAD_INDEX); return; }
  st.cur_len[b] = seg_pos0[i] + seg_rows[i];
  st.len0[b] = st.cur_len[b];
  st.active[b] = 0;
}

__global__ void feed_kernel(StepState st, const int* seqs, const int* tokens, int n) {
  pdl_launch_dependents();
  pdl_wait();
  for (int b = threadIdx.x; b < st.n_seqs; b += blockDim.x) st.active[b] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int b = seqs[i];
    if (b < 0 || b >= st.n_seqs) { arcb_set_error(st.err, ARCB_DEV_BAD_INDEX); continue; }
    st.active[b] = 1;
    st.cur_tok[b] = tokens[i];
  }
}

__global__ void pack_blocks_kernel(const float* __restrict__ src, void* __restrict__ dst, long long rows, long long cols,
                                   int rb, int rbp, int row_off, int cb, int cbp, long long dst_pitch, int container) {
  const long long n = rows * cols;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / cols, c = i - r * cols;
    const long long at = (row_off + (r / rb) * rbp + r % rb) * dst_pitch + (c / cb) * cbp + c % cb;
    if (container == 2) reinterpret_cast<float*>(dst)[at] = src[i];
    else st_act(dst, at, __bfloat162float(__float2bfloat16_rn(src[i])), container);
  }
}

__global__ void pack_heads_t_kernel(const float* __restrict__ src, void* __restrict__ dst, int heads, int rb, int rbp, int cols,
                                    long long dst_pitch, int container) {
  const long long n = (long long)heads * rb * cols;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / cols;
    const int c = (int)(i - r * cols), h = (int)(r / rb), d = (int)(r - (long long)h * rb);
    const long long at = ((long long)h * rbp + c) * dst_pitch + d;
    if (container == 2) reinterpret_cast<float*>(dst)[at] = src[i];
    else st_act(dst, at, __bfloat162float(__float2bfloat16_rn(src[i])), container);
  }
}

}  // namespace

int arcb_launch_sandwich_norm(const SandwichArgs& a, cudaStream_t stream) {
  if (a.rows <= 0) return 0;
  if (a.pitch % 128) return -1;
  const dim3 grid(a.rows), block(128);
  const int steps = (a.pitch + 511) / 512;
  const bool ahead = a.rows <= 1024;
  auto go = [&](auto few, auto many) { return arcb_launch(ahead ? few : many, grid, block, 0, stream, a); };
  const cudaError_t e = steps <= 2   ? go(sandwich_norm_kernel<2, true, true>, sandwich_norm_kernel<2, true, false>)
                        : steps <= 3 ? go(sandwich_norm_kernel<3, true, true>, sandwich_norm_kernel<3, true, false>)
                        : steps <= 4 ? go(sandwich_norm_kernel<4, true, true>, sandwich_norm_kernel<4, true, false>)
                        : steps <= 8 ? go(sandwich_norm_kernel<8, true, true>, sandwich_norm_kernel<8, true, false>)
                                     : arcb_launch(sandwich_norm_kernel<1, false, false>, grid, block, 0, stream, a);
  arcb_count_launch(1);
  return (int)e;
}

int arcb_launch_latent_prep(const LatentPrepArgs& a, cudaStream_t stream) {
  if (a.rows <= 0) return 0;
  if (a.q_rankp % 4 || a.kv_rankp % 64 || a.rotp % 64 || a.pitch % 4 || a.off_c != a.q_rankp || a.off_r != a.off_c + a.kv_rankp) return -1;
  const int steps = (a.off_r + a.rotp + 511) / 512;
  const dim3 grid(a.rows), block(128);
  const cudaError_t e = steps <= 1   ? arcb_launch(latent_prep_kernel<1>, grid, block, 0, stream, a)
                        : steps <= 3 ? arcb_launch(latent_prep_kernel<3>, grid, block, 0, stream, a)
                        : steps <= 6 ? arcb_launch(latent_prep_kernel<6>, grid, block, 0, stream, a)
                        : steps <= 12 ? arcb_launch(latent_prep_kernel<12>, grid, block, 0, stream, a)
                                      : cudaErrorInvalidValue;
  arcb_count_launch(1);
  return (int)e;
}

int arcb_launch_rot_table(float2* table, int t_max, int pairs, int dims, double base, cudaStream_t stream) {
  if (t_max <= 0 || pairs <= 0) return 0;
  long long blocks = ((long long)t_max * pairs + 255) / 256;
  if (blocks > 148 * 8) blocks = 148 * 8;
  rot_table_kernel<<<(unsigned)blocks, 256, 0, stream>>>(table, t_max, pairs, dims, base);
  arcb_count_launch(1);
  return (int)cudaGetLastError();
}

int arcb_launch_pack_heads_t(const float* src, void* dst, int heads, int rb, int rbp, int cols, long long dst_pitch, int container,
                             cudaStream_t stream) {
  const long long n = (long long)heads * rb * cols;
  if (n <= 0) return 0;
  long long blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  pack_heads_t_kernel<<<(unsigned)blocks, 256, 0, stream>>>(src, dst, heads, rb, rbp, cols, dst_pitch, container);
  arcb_count_launch(1);
  return (int)cudaGetLastError();
}

int arcb_launch_lm_embed(const LmEmbedArgs& a, cudaStream_t stream) {
  if (a.rows <= 0) return 0;
  const cudaError_t e = arcb_launch(lm_embed_kernel, dim3((a.rows + ROWS_PER_CTA - 1) / ROWS_PER_CTA), dim3(ROWS_PER_CTA * 32), 0, stream, a);
  arcb_count_launch(1);
  return (int)e;
}

int arcb_launch_step_begin(const StepState& st, const LmEmbedArgs& a, cudaStream_t stream) {
  const cudaError_t e = arcb_launch(step_begin_kernel, dim3((st.n_seqs + ROWS_PER_CTA - 1) / ROWS_PER_CTA), dim3(ROWS_PER_CTA * 32), 0, stream, st, a);
  arcb_count_launch(1);
  return (int)e;
}

int arcb_launch_lm_norm(const LmNormArgs& a, cudaStream_t stream) {
  if (a.rows <= 0) return 0;
  if (a.pitch % 128) return -1;
  const cudaError_t e = arcb_launch(lm_norm_kernel, dim3((a.rows + ROWS_PER_CTA - 1) / ROWS_PER_CTA), dim3(ROWS_PER_CTA * 32), 0, stream, a);
  arcb_count_launch(1);
  return (int)e;
}

int arcb_launch_proj_prep(const ProjArgs& a, const float* proj, cudaStream_t stream) {
  if (a.M <= 0) return 0;
  const int nkv = a.recurrent ? a.H : a.G;
  const int units = 2 * a.H + (a.off_k >= 0 ? 2 * nkv : 0) + (a.recurrent ? 1 : 0);
  const long long blocks = ((long long)a.M * units + 3) / 4;
  if (blocks > 0x7fffffffLL) return -1;
  const cudaError_t e = arcb_launch(proj_prep_kernel, dim3((unsigned)blocks), dim3(128), 0, stream, a, proj, units);
  arcb_count_launch(1);
  return (int)e;
}

int arcb_launch_pick(const PickArgs& a, const StepState& st, cudaStream_t stream) {
  if (a.rows <= 0) return 0;
  const cudaError_t e = arcb_launch(pick_kernel, dim3(a.rows), dim3(PICK_THREADS), 0, stream, a, st);
  arcb_count_launch(1);
  return (int)e;
}

int arcb_launch_seg_commit(const StepState& st, const int* seg_seq, const int* seg_pos0, const int* seg_rows, int n,
                           cudaStream_t stream) {
  if (n <= 0) return 0;
  const cudaError_t e = arcb_launch(seg_commit_kernel, dim3((n + 127) / 128), dim3(128), 0, stream, st, seg_seq, seg_pos0, seg_rows, n);
  arcb_count_launch(1);
  return (int)e;
}

int arcb_launch_feed(const StepState& st, const int* seqs, const int* tokens, int n, cudaStream_t stream) {
  const cudaError_t e = arcb_launch(feed_kernel, dim3(1), dim3(256), 0, stream, st, seqs, tokens, n);
  arcb_count_launch(1);
  return (int)e;
}

int arcb_launch_pack_blocks(const float* src, void* dst, long long rows, long long cols, int rb, int rbp, int row_off,
                            int cb, int cbp, long long dst_pitch, int container, cudaStream_t stream) {
  const long long n = rows * cols;
  if (n <= 0) return 0;
  long long blocks = (n + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  pack_blocks_kernel<<<(unsigned)blocks, 256, 0, stream>>>(src, dst, rows, cols, rb, rbp, row_off, cb, cbp, dst_pitch, container);
  arcb_count_launch(1);
  return (int)cudaGetLastError();
}
