// Kernel template of the grouped-head streaming attention.
//
// One CTA of four warps owns one (query row, key/value head, tile of up to four of its query heads,
// split).  The warps take alternating slices of the cached prefix.  Inside a warp LPR lanes share one
// key: each lane holds DE query dims of every query head of the tile and VE value dims of the
// accumulators, so a key (value) row is loaded once, 16 bytes a lane, and used for all heads of the
// tile.  Partial scores are reduced by a transposing butterfly: after it every lane holds the complete
// score of ONE head of the tile (head = (lane % LPR) / (LPR / RT)), so exponentials, maxima and sums
// are computed once per (key, head) and the weights are handed back by shuffles.  Scores, weights and
// sums are fp32.  Warps merge through shared memory in a fixed order.
#pragma once
#include "attn_gqa.cuh"
#include "launch.cuh"

namespace {

constexpr int GQA_WARPS = 4;
#ifndef ARCB_GQA_STEPS
#define ARCB_GQA_STEPS 4
#endif
constexpr int GQA_STEPS = ARCB_GQA_STEPS;   // most load steps in flight per warp and plane
constexpr float GQA_LOG2E = 1.4426950408889634f;

__host__ __device__ constexpr int gqa_max(int a, int b) { return a > b ? a : b; }
__host__ __device__ constexpr int gqa_min(int a, int b) { return a < b ? a : b; }
// lanes that share one key: 16 bytes a lane of the wider of the two rows
__host__ __device__ constexpr int gqa_lpr(int fmt, int dp, int vp) { return gqa_min(32, gqa_max(dp, vp) * (fmt == 2 ? 4 : 2) / 16); }

// two fp32 values in one 64-bit register pair, and the two-wide multiply-add on them
__device__ __forceinline__ uint64_t f2_pack(float lo, float hi) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 f2_unpack(uint64_t v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ uint64_t f2_fma(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t f2_mul(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// 2 N consecutive elements -> N fp32 pairs
template <int FMT, int N>
__device__ __forceinline__ void gqa_unpack(const uint32_t* raw, uint64_t (&out)[N]) {
#pragma unroll
  for (int i = 0; i < N; ++i) {
    if constexpr (FMT == 2) {
      out[i] = f2_pack(__uint_as_float(raw[2 * i]), __uint_as_float(raw[2 * i + 1]));
    } else {
      const float2 f = unpack2_act(raw[i], FMT);
      out[i] = f2_pack(f.x, f.y);
    }
  }
}

// W 32-bit words from global memory (16- or 8-byte loads, no L1 allocation)
template <int W>
__device__ __forceinline__ void gqa_load(const void* p, uint32_t (&r)[W]) {
  if constexpr (W % 4 == 0) {
#pragma unroll
    for (int i = 0; i < W / 4; ++i) {
      const uint4 t = ldg_stream16(reinterpret_cast<const uint4*>(p) + i);
      r[4 * i] = t.x; r[4 * i + 1] = t.y; r[4 * i + 2] = t.z; r[4 * i + 3] = t.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < W / 2; ++i) {
      const uint2 t = __ldg(reinterpret_cast<const uint2*>(p) + i);
      r[2 * i] = t.x; r[2 * i + 1] = t.y;
    }
    if constexpr (W % 2) r[W - 1] = __ldg(reinterpret_cast<const uint32_t*>(p) + W - 1);
  }
}

template <int FMT, int DP, int VP, int RT>
__global__ void __launch_bounds__(GQA_WARPS * 32)
attn_gqa_kernel(AttnGqaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int ES = FMT == 2 ? 4 : 2;
  constexpr int LPR = gqa_lpr(FMT, DP, VP);
  constexpr int DE = DP / LPR, VE = VP / LPR;            // dims per lane
  constexpr int KW = DE * ES / 4, VW = VE * ES / 4;      // 32-bit words per lane and row
  constexpr int RPL = 32 / LPR;                          // rows per load step
  constexpr int U = gqa_max(1, gqa_min(GQA_STEPS, 32 / gqa_max(KW, VW)));   // load steps per iteration
  constexpr int ROWS = U * RPL;
  constexpr int REC = VP + 4;
  __shared__ float s_part[GQA_WARPS][RT][REC];

  const int lane = threadIdx.x & 31, wj = threadIdx.x >> 5;
  long long w = blockIdx.x;
  const int split = (int)(w % a.n_splits); w /= a.n_splits;
  const int tile = (int)(w % a.tiles); w /= a.tiles;
  const int g = (int)(w % a.n_kv);
  const int item = (int)(w / a.n_kv);
  const int h0 = g * a.rep + tile * a.tile_rows;                       // first query head of the tile
  const int nh = min(a.tile_rows, a.rep - tile * a.tile_rows);         // heads in the tile (<= RT)

  const int seq = a.item_seq ? a.item_seq[item] : item;
  int len = a.item_len[item];
  if (len > a.t_max || seq < 0 || seq >= a.n_seqs) {
    if (threadIdx.x == 0) arcb_set_error(a.err, ARCB_DEV_BAD_INDEX);
    len = 0;
  }
  if (len < 0) len = 0;
  int begin = 0, end = len;
  if (a.n_splits > 1) {
    int chunk = (len + a.n_splits - 1) / a.n_splits;
    chunk = (chunk + 15) & ~15;
    begin = min(split * chunk, len);
    end = min(begin + chunk, len);
  }

  const int sub = lane / LPR, seg = lane % LPR;
  const int my_r = seg / (LPR / RT);                     // head whose scores this lane keeps
  uint64_t q[RT][DE / 2];
#pragma unroll
  for (int r = 0; r < RT; ++r) {
    const float sc = r < nh ? a.scale * GQA_LOG2E : 0.f;
    const int h = h0 + min(r, nh - 1);
#pragma unroll
    for (int e = 0; e < DE / 2; ++e) {
      const size_t at = (size_t)item * a.q_pitch + (size_t)h * DP + seg * DE + 2 * e;
      q[r][e] = f2_pack(ld_act(a.q, at, FMT) * sc, ld_act(a.q, at + 1, FMT) * sc);
    }
  }
  const size_t row0 = ((size_t)seq * a.n_kv + g) * (size_t)a.t_max;
  const char* Kp = reinterpret_cast<const char*>(a.k) + (row0 * DP + seg * DE) * ES;
  const char* Vp = reinterpret_cast<const char*>(a.v) + (row0 * VP + seg * VE) * ES;

  float m = -INFINITY, l = 0.f;                          // of head my_r, this lane group's rows
  uint64_t acc[RT][VE / 2];
#pragma unroll
  for (int r = 0; r < RT; ++r)
#pragma unroll
    for (int e = 0; e < VE / 2; ++e) acc[r][e] = 0ull;

  for (int r0 = begin + wj * ROWS; r0 < end; r0 += ROWS * GQA_WARPS) {
    uint32_t kk[U][KW], vv[U][VW];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int row = r0 + u * RPL + sub;
#pragma unroll
      for (int i = 0; i < KW; ++i) kk[u][i] = 0u;
      if (row < end) gqa_load<KW>(Kp + (size_t)row * (DP * ES), kk[u]);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int row = r0 + u * RPL + sub;
#pragma unroll
      for (int i = 0; i < VW; ++i) vv[u][i] = 0u;
      if (row < end) gqa_load<VW>(Vp + (size_t)row * (VP * ES), vv[u]);
    }
    float s[U];
    float mx = m;
#pragma unroll
    for (int u = 0; u < U; ++u) {
      uint64_t kf[DE / 2];
      gqa_unpack<FMT, DE / 2>(kk[u], kf);
      float d[RT];
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        uint64_t d2 = f2_mul(q[r][0], kf[0]);
#pragma unroll
        for (int e = 1; e < DE / 2; ++e) d2 = f2_fma(q[r][e], kf[e], d2);
        const float2 f = f2_unpack(d2);
        d[r] = f.x + f.y;
      }
      // transposing butterfly: RT partial sums -> one complete sum per lane
#pragma unroll
      for (int st = RT / 2; st >= 1; st >>= 1) {
        const int dist = (LPR / RT) * st;
        const bool up = (lane & dist) != 0;
#pragma unroll
        for (int j = 0; j < st; ++j) {
          const float send = up ? d[j] : d[j + st];
          const float keep = up ? d[j + st] : d[j];
          d[j] = keep + __shfl_xor_sync(0xffffffffu, send, dist);
        }
      }
#pragma unroll
      for (int dist = LPR / RT / 2; dist >= 1; dist >>= 1) d[0] += __shfl_xor_sync(0xffffffffu, d[0], dist);
      s[u] = (r0 + u * RPL + sub < end) ? d[0] : -INFINITY;
      mx = fmaxf(mx, s[u]);
    }
    const float m_safe = (mx == -INFINITY) ? 0.f : mx;
    const float alpha = exp2f(m - m_safe);
    l *= alpha;
    m = mx;
#pragma unroll
    for (int r = 0; r < RT; ++r) {
      const float al = RT == 1 ? alpha : __shfl_sync(0xffffffffu, alpha, sub * LPR + r * (LPR / RT));
      const uint64_t al2 = f2_pack(al, al);
#pragma unroll
      for (int e = 0; e < VE / 2; ++e) acc[r][e] = f2_mul(acc[r][e], al2);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const float p = exp2f(s[u] - m_safe);
      l += p;
      uint64_t vf[VE / 2];
      gqa_unpack<FMT, VE / 2>(vv[u], vf);
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        const float pr = RT == 1 ? p : __shfl_sync(0xffffffffu, p, sub * LPR + r * (LPR / RT));
        const uint64_t pr2 = f2_pack(pr, pr);
#pragma unroll
        for (int e = 0; e < VE / 2; ++e) acc[r][e] = f2_fma(pr2, vf[e], acc[r][e]);
      }
    }
  }

  // merge the lane groups of the warp (lanes LPR apart hold the same dims and the same head)
#pragma unroll
  for (int o = LPR; o < 32; o <<= 1) {
    const float m_o = __shfl_xor_sync(0xffffffffu, m, o);
    const float l_o = __shfl_xor_sync(0xffffffffu, l, o);
    const float mx = fmaxf(m, m_o);
    const float m_safe = (mx == -INFINITY) ? 0.f : mx;
    const float sa = exp2f(m - m_safe), sb = exp2f(m_o - m_safe);
    l = l * sa + l_o * sb;
    m = mx;
#pragma unroll
    for (int r = 0; r < RT; ++r) {
      const int src = sub * LPR + r * (LPR / RT);
      const float ra = __shfl_sync(0xffffffffu, sa, src), rb = __shfl_sync(0xffffffffu, sb, src);
#pragma unroll
      for (int e = 0; e < VE / 2; ++e) {
        const float2 mine = f2_unpack(acc[r][e]);
        const float ox = __shfl_xor_sync(0xffffffffu, mine.x, o), oy = __shfl_xor_sync(0xffffffffu, mine.y, o);
        acc[r][e] = f2_pack(mine.x * ra + ox * rb, mine.y * ra + oy * rb);
      }
    }
  }
  if (sub == 0) {
#pragma unroll
    for (int r = 0; r < RT; ++r)
#pragma unroll
      for (int e = 0; e < VE / 2; ++e)
        *reinterpret_cast<float2*>(&s_part[wj][r][seg * VE + 2 * e]) = f2_unpack(acc[r][e]);
    if (seg % (LPR / RT) == 0) {
      s_part[wj][my_r][VP] = m;
      s_part[wj][my_r][VP + 1] = l;
    }
  }
  __syncthreads();
  // every warp finishes the heads wj, wj + 4, ... of the tile: warps merged in a fixed order
  for (int r = wj; r < nh; r += GQA_WARPS) {
    float mt = -INFINITY;
#pragma unroll
    for (int j = 0; j < GQA_WARPS; ++j) mt = fmaxf(mt, s_part[j][r][VP]);
    const int h = h0 + r;
    const bool last = a.n_splits == 1;
    const float sk = (last && a.sink) ? a.sink[h] * GQA_LOG2E : -INFINITY;
    if (last) mt = fmaxf(mt, sk);
    const float mt_safe = (mt == -INFINITY) ? 0.f : mt;
    float sc[GQA_WARPS], lt = exp2f(sk - mt_safe);
#pragma unroll
    for (int j = 0; j < GQA_WARPS; ++j) {
      sc[j] = exp2f(s_part[j][r][VP] - mt_safe);
      lt += s_part[j][r][VP + 1] * sc[j];
    }
    const float inv = lt > 0.f ? 1.f / lt : 0.f;
    const size_t oh = (size_t)item * a.n_heads + h;
    for (int c = lane; c < VP; c += 32) {
      float o = 0.f;
#pragma unroll
      for (int j = 0; j < GQA_WARPS; ++j) o += s_part[j][r][c] * sc[j];
      if (last) {
        o *= inv;
        if (a.gate) o *= ld_act(a.gate, (size_t)item * a.gate_pitch + (size_t)h * VP + c, FMT);
        st_act(a.out, oh * VP + c, o, FMT);
      } else {
        a.scratch[(oh * a.n_splits + split) * REC + c] = o;
      }
    }
    if (!last && lane == 0) {
      float* rec = a.scratch + (oh * a.n_splits + split) * REC;
      rec[VP] = mt;
      rec[VP + 1] = lt;
    }
  }
}

template <int FMT, int DP, int VP>
cudaError_t gqa_launch_dv(const AttnGqaArgs& a, dim3 grid, cudaStream_t stream) {
  constexpr int LPR = gqa_lpr(FMT, DP, VP);
  static_assert(LPR >= 4, "a key spans at least four lanes");
  if (a.tile_rows == 1) return arcb_launch(attn_gqa_kernel<FMT, DP, VP, 1>, grid, dim3(GQA_WARPS * 32), 0, stream, a);
  if (a.tile_rows == 2) return arcb_launch(attn_gqa_kernel<FMT, DP, VP, 2>, grid, dim3(GQA_WARPS * 32), 0, stream, a);
  return arcb_launch(attn_gqa_kernel<FMT, DP, VP, 4>, grid, dim3(GQA_WARPS * 32), 0, stream, a);
}

template <int FMT>
cudaError_t gqa_dispatch(const AttnGqaArgs& a, dim3 grid, cudaStream_t stream) {
  switch (a.dimp * 1000 + a.vdimp) {
    case 64064: return gqa_launch_dv<FMT, 64, 64>(a, grid, stream);
    case 64128: return gqa_launch_dv<FMT, 64, 128>(a, grid, stream);
    case 64256: return gqa_launch_dv<FMT, 64, 256>(a, grid, stream);
    case 128064: return gqa_launch_dv<FMT, 128, 64>(a, grid, stream);
    case 128128: return gqa_launch_dv<FMT, 128, 128>(a, grid, stream);
    case 128256: return gqa_launch_dv<FMT, 128, 256>(a, grid, stream);
    case 256064: return gqa_launch_dv<FMT, 256, 64>(a, grid, stream);
    case 256128: return gqa_launch_dv<FMT, 256, 128>(a, grid, stream);
    case 256256: return gqa_launch_dv<FMT, 256, 256>(a, grid, stream);
  }
  return cudaErrorInvalidValue;
}

}  // namespace
