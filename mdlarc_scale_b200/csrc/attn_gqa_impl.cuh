// Kernel template of the grouped-head streaming attention.
//
// One CTA of four warps owns one (query row, key/value head, tile of up to four of its query heads,
// split).  The warps take alternating slices of the cached prefix.  Inside a warp LPR lanes share one
// key: each lane holds DE query dims of every query head of the tile and VE value dims of the
// accumulators, so a key (value) row is loaded once, 16 bytes a lane, and used for all heads of the
// tile.  Rows are copied asynchronously into a ring in shared memory several stages ahead; a lane reads back only
// the bytes it copied itself, so the ring needs no barrier, and the bytes in flight cost no registers.
// Partial scores are reduced by a transposing butterfly: after it every lane holds the complete
// score of ONE head of the tile (head = (lane % LPR) / (LPR / RT)), so exponentials, maxima and sums
// are computed once per (key, head) and the weights are handed back by shuffles.  Scores, weights and
// sums are fp32.  Warps merge through shared memory in a fixed order.
#pragma once
#include "attn_gqa.cuh"
#include "launch.cuh"

namespace {

constexpr int GQA_WARPS = 4;
#ifndef ARCB_GQA_STAGES
#define ARCB_GQA_STAGES 3
#endif
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

// W 32-bit words, global -> shared, zeros when !valid
template <int W>
__device__ __forceinline__ void gqa_copy(uint32_t dst, const void* src, bool valid) {
  if constexpr (W % 4 == 0) {
#pragma unroll
    for (int i = 0; i < W / 4; ++i)
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + i * 512), "l"(reinterpret_cast<const char*>(src) + i * 16),
                   "r"(valid ? 16 : 0) : "memory");
  } else if constexpr (W == 2) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(dst), "l"(src), "r"(valid ? 8 : 0) : "memory");
  } else {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(dst), "l"(src), "r"(valid ? 4 : 0) : "memory");
  }
}
template <int W>
__device__ __forceinline__ void gqa_fetch(const uint8_t* src, uint32_t (&r)[W]) {
  if constexpr (W % 4 == 0) {
#pragma unroll
    for (int i = 0; i < W / 4; ++i) {
      const uint4 t = *reinterpret_cast<const uint4*>(src + i * 512);
      r[4 * i] = t.x; r[4 * i + 1] = t.y; r[4 * i + 2] = t.z; r[4 * i + 3] = t.w;
    }
  } else if constexpr (W == 2) {
    const uint2 t = *reinterpret_cast<const uint2*>(src);
    r[0] = t.x; r[1] = t.y;
  } else {
    r[0] = *reinterpret_cast<const uint32_t*>(src);
  }
}

// Sizes of one instantiation.  A slot is what a warp loads of one plane in one step (its lanes' words side by
// side, 16 bytes a lane at most); a stage is U slots of keys and U of values.
template <int FMT, int DP, int VP>
struct GqaCfg {
  static constexpr int ES = FMT == 2 ? 4 : 2;
  static constexpr int LPR = gqa_lpr(FMT, DP, VP);
  static constexpr int DE = DP / LPR, VE = VP / LPR;            // dims per lane
  static constexpr int KW = DE * ES / 4, VW = VE * ES / 4;      // 32-bit words per lane and row
  static constexpr int RPL = 32 / LPR;                          // rows per load step
  static constexpr int U = gqa_max(KW, VW) > 4 ? 2 : 4;         // load steps per stage
  static constexpr int ROWS = U * RPL;
  static constexpr int K_SLOT = 128 * KW, V_SLOT = 128 * VW;
  static constexpr int STAGE = U * (K_SLOT + V_SLOT);
  static constexpr int STAGES = ARCB_GQA_STAGES;
  static constexpr int SMEM = GQA_WARPS * STAGES * STAGE;
};

template <int FMT, int DP, int VP, int RT>
__global__ void __launch_bounds__(GQA_WARPS * 32)
attn_gqa_kernel(AttnGqaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  using C = GqaCfg<FMT, DP, VP>;
  constexpr int ES = C::ES, LPR = C::LPR, DE = C::DE, VE = C::VE, KW = C::KW, VW = C::VW, RPL = C::RPL, U = C::U, ROWS = C::ROWS;
  constexpr int REC = VP + 4;
  static_assert(C::SMEM >= GQA_WARPS * RT * REC * 4, "the warps' partial results reuse the ring");
  extern __shared__ __align__(16) uint8_t gqa_smem[];
  float (*s_part)[RT][REC] = reinterpret_cast<float (*)[RT][REC]>(gqa_smem);

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
  int begin = a.window > 0 ? max(0, len - a.window) : 0, end = len;
  if (a.n_splits > 1) {
    int chunk = (len - begin + a.n_splits - 1) / a.n_splits;
    chunk = (chunk + 15) & ~15;
    begin = min(begin + split * chunk, len);
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

  uint8_t* ring = gqa_smem + wj * (C::STAGES * C::STAGE);
  const uint32_t ring_addr = static_cast<uint32_t>(__cvta_generic_to_shared(ring));
  constexpr int K_LANE = KW % 4 == 0 ? 16 : KW * 4, V_LANE = VW % 4 == 0 ? 16 : VW * 4;   // distance between lanes in a slot
  auto issue = [&](int r0, int stage) {     // every lane commits, also past the end: the group count stays in step
    const uint32_t st = ring_addr + stage * C::STAGE;
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int row = r0 + u * RPL + sub;
      const bool ok = row < end;
      gqa_copy<KW>(st + u * C::K_SLOT + lane * K_LANE, Kp + (size_t)(ok ? row : 0) * (DP * ES), ok);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int row = r0 + u * RPL + sub;
      const bool ok = row < end;
      gqa_copy<VW>(st + U * C::K_SLOT + u * C::V_SLOT + lane * V_LANE, Vp + (size_t)(ok ? row : 0) * (VP * ES), ok);
    }
  };
  constexpr int STEP = ROWS * GQA_WARPS;
  int ahead = begin + wj * ROWS;            // first row of the next stage to issue
  int put = 0, get = 0;
#pragma unroll
  for (int i = 0; i < C::STAGES - 1; ++i) {
    if (ahead < end) issue(ahead, put);
    asm volatile("cp.async.commit_group;" ::: "memory");
    ahead += STEP;
    ++put;
  }
  for (int r0 = begin + wj * ROWS; r0 < end; r0 += STEP) {
    if (ahead < end) issue(ahead, put);
    asm volatile("cp.async.commit_group;" ::: "memory");
    ahead += STEP;
    put = put + 1 == C::STAGES ? 0 : put + 1;
    asm volatile("cp.async.wait_group %0;" ::"n"(C::STAGES - 1) : "memory");
    const uint8_t* slot = ring + get * C::STAGE;
    get = get + 1 == C::STAGES ? 0 : get + 1;
    float s[U];
    float mx = m;
#pragma unroll
    for (int u = 0; u < U; ++u) {
      uint32_t kw[KW];
      gqa_fetch<KW>(slot + u * C::K_SLOT + lane * K_LANE, kw);
      uint64_t kf[DE / 2];
      gqa_unpack<FMT, DE / 2>(kw, kf);
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
    if (__any_sync(0xffffffffu, alpha != 1.f)) {
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        const float al = RT == 1 ? alpha : __shfl_sync(0xffffffffu, alpha, sub * LPR + r * (LPR / RT));
        const uint64_t al2 = f2_pack(al, al);
#pragma unroll
        for (int e = 0; e < VE / 2; ++e) acc[r][e] = f2_mul(acc[r][e], al2);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const float p = exp2f(s[u] - m_safe);
      l += p;
      uint32_t vw[VW];
      gqa_fetch<VW>(slot + U * C::K_SLOT + u * C::V_SLOT + lane * V_LANE, vw);
      uint64_t vf[VE / 2];
      gqa_unpack<FMT, VE / 2>(vw, vf);
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
  __syncthreads();     // every warp is done with its ring
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

template <int FMT, int DP, int VP, int RT>
cudaError_t gqa_launch_one(const AttnGqaArgs& a, dim3 grid, cudaStream_t stream) {
  using C = GqaCfg<FMT, DP, VP>;
  if (C::SMEM > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(attn_gqa_kernel<FMT, DP, VP, RT>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM);
    if (e != cudaSuccess) return e;
  }
  return arcb_launch(attn_gqa_kernel<FMT, DP, VP, RT>, grid, dim3(GQA_WARPS * 32), C::SMEM, stream, a);
}

template <int FMT, int DP, int VP>
cudaError_t gqa_launch_dv(const AttnGqaArgs& a, dim3 grid, cudaStream_t stream) {
  static_assert(GqaCfg<FMT, DP, VP>::LPR >= 4, "a key spans at least four lanes");
  if (a.tile_rows == 1) return gqa_launch_one<FMT, DP, VP, 1>(a, grid, stream);
  if (a.tile_rows == 2) return gqa_launch_one<FMT, DP, VP, 2>(a, grid, stream);
  return gqa_launch_one<FMT, DP, VP, 4>(a, grid, stream);
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
