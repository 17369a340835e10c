// Chunkwise prefill of the matrix-memory recurrence on tensor cores.
//
// One CTA owns one (segment, head) and walks the segment in chunks of 64 tokens with the fp32 state in
// registers.  Inside a chunk, with F_t the running sum of the log forget gates, c_s = i_s - F_s and
// M_t = max(m, max_{s <= t} c_s) (m: stabiliser at the chunk's start), the recurrence unrolls to
//   m_t   = F_t + M_t
//   num_t = exp(m - M_t) S^T q_t + sum_{s <= t} exp(c_s - M_t) (q_t . k_s) v_s
//   n.q_t = exp(m - M_t) n . q_t + sum_{s <= t} exp(c_s - M_t) (q_t . k_s)
//   S'    = exp(m - M_L) S + sum_s exp(c_s - M_L) k_s v_s^T         (n alike)
// so every exponent is at most zero and the result is the token-by-token one up to rounding.
//
// The state is held as S^T: warp w owns value rows [16 w, 16 w + 16) of all key columns as MMA accumulators,
// whose registers are at the same time, pairwise packed, the B operand of Q S.  Products that read or add to
// the state use operands split into a rounded part and its remainder, so the state keeps close to fp32
// precision; the decay-weighted scores are rounded once to the operand format, like attention weights.
// A producer warp issues the TMA loads (64 x 64 boxes, 128-byte swizzle) one chunk ahead and evaluates the next
// chunk's gates while the other warps compute; the output gates replace the queries in their tile once those
// have been read.  The products are small (64 rows) and the launch is bound by reading q, k, v and the gates,
// so warp-level MMA is enough to stay near that bound.
#include "flash_common.cuh"
#include "gemm.cuh"
#include "launch.cuh"
#include "mlstm.cuh"
#include "ptx_sm100.cuh"

using namespace sm100;

namespace {

constexpr int L = 64;      // tokens per chunk
constexpr float LOG2E = 1.4426950408889634f;

// CTAs per SM the register and shared-memory budgets are set for, and the registers of a computing thread after
// the helper warpgroup has given up its own (24 each): helper + computing registers fit what a launch of that
// many CTAs is given (checked against the compiled kernel in arcb_mlstm_chunk_init)
__host__ __device__ constexpr int chunk_ctas(int d, int vp) { return vp == 128 ? (d == 128 ? 1 : 2) : (d == 128 ? 2 : 3); }
__host__ __device__ constexpr int chunk_regs(int d, int vp) { return vp == 128 ? (d == 128 ? 240 : 104) : (d == 128 ? 232 : 136); }

template <int R>
__device__ __forceinline__ void reg_alloc() { asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(R)); }

__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
template <bool F16>
__device__ __forceinline__ void mma16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  if constexpr (F16)
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
  else
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <bool F16>
__device__ __forceinline__ uint32_t pack2_raw(float x, float y) {
  if constexpr (F16) {
    const __half2 h = __floats2half2_rn(x, y);
    return *reinterpret_cast<const uint32_t*>(&h);
  } else {
    return pack2_bf16(x, y);
  }
}
// (x, y) as a packed pair and the packed pair of what the rounding left over
template <bool F16>
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack2_raw<F16>(x, y);
  const float2 h = unpack2_act(hi, F16 ? 1 : 0);
  lo = pack2_raw<F16>(x - h.x, y - h.y);
}

// byte offset of 16-byte chunk `ch` of row `row` in a tile made of L-row x 64-column boxes (TMA's 128-byte swizzle)
__device__ __forceinline__ uint32_t tile_off(int row, int ch) {
  return (uint32_t)((ch >> 3) * (L * 128) + row * 128 + (((ch & 7) ^ (row & 7)) << 4));
}

template <int D, int VP>
struct ChunkCfg {
  static constexpr int NW = VP / 16;         // computing warps
  static constexpr int NC = NW * 32;         // computing threads
  static constexpr int NT = NC + 128;        // and a helper warpgroup, whose first warp is the producer
  static constexpr int NB = NC + 32;         // threads of the chunk barrier
  static constexpr int QB = L * D * 2, VB = L * VP * 2;
  static constexpr int Q_TILE = QB > VB ? QB : VB;   // queries, then output gates
  static constexpr int STAGE = Q_TILE + QB + VB;     // q / gates, k, v
  static constexpr int PB = L * L * 2;
  static constexpr int GATE_FLOATS = 5 * L + 2;      // c, M, w, row factor, exp(-m_t); exp(m - M_L), m at the end
  // stages | P | gates x 2 | n.q | score sums [2][L] | n [D] | n partials [4][D] | squares [NW][L]
  static constexpr int FLOATS = 2 * GATE_FLOATS + 3 * L + 5 * D + NW * L;
  static constexpr int SMEM = 2 * STAGE + PB + FLOATS * 4 + 64 + 1024;
};

template <bool F16, int D, int VP>
__global__ void __launch_bounds__(ChunkCfg<D, VP>::NT, chunk_ctas(D, VP))
mlstm_chunk_kernel(const __grid_constant__ CUtensorMap tmap, MlstmArgs a) {
  using C = ChunkCfg<D, VP>;
  constexpr int NW = C::NW, NC = C::NC;
  constexpr int KH = NW / 4;                 // key halves of the score blocks
  constexpr float S_SCALE = F16 ? 1.f / 256.f : 1.f;   // keeps long sums of the state inside the half range
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* bp = smem_raw + (base - raw);
  const uint32_t p_smem = base + 2 * C::STAGE;
  float* f_gate = reinterpret_cast<float*>(bp + 2 * C::STAGE + C::PB);
  float* f_qn = f_gate + 2 * C::GATE_FLOATS;   // n . q_t of the carried state
  float* f_sum = f_qn + L;       // [KH <= 2][L] score sums
  float* f_n = f_sum + 2 * L;    // [D]
  float* f_np = f_n + D;         // [4][D]
  float* f_ss = f_np + 4 * D;    // [NW][L]
  const uint32_t bars = base + 2 * C::STAGE + C::PB + ((C::FLOATS * 4 + 15) & ~15);   // full[2], output gates

  // warps 0-3: helpers (the first is the producer); computing warps count from 0 behind them
  const bool helper = threadIdx.x < 128, producer = threadIdx.x < 32;
  const int tid = helper ? (int)threadIdx.x : (int)threadIdx.x - 128, lane = tid & 31, warp = tid >> 5;
  const int g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.x, sg = blockIdx.y;
  const int row0 = a.seg_row0[sg], rows = a.seg_rows[sg], seq = a.seg_seq[sg];
  const bool fresh = a.seg_pos0[sg] == 0;
  if (seq < 0 || seq >= a.n_seqs) {
    if (tid == 0) arcb_set_error(a.err, ARCB_DEV_BAD_INDEX);
    return;
  }
  if (rows <= 0) return;
  float* Sg = a.S + ((size_t)seq * a.H + h) * a.dim * VP;
  float* ng = a.n + ((size_t)seq * a.H + h) * a.dimp;
  float* mg = a.m + (size_t)seq * a.H + h;
  const int v_lo = warp * 16 + g;            // this lane's value rows: v_lo and v_lo + 8

  for (int d = threadIdx.x; d < D; d += C::NT) f_n[d] = (!fresh && d < a.dim) ? ng[d] : 0.f;
  float m = fresh ? 0.f : *mg;

  const int n_chunks = (rows + L - 1) / L;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(bars + 8 * i, 1);
    mbar_fence_init();
    tma_prefetch_desc(&tmap);
  }
  __syncthreads();
  if (helper) reg_dealloc_24();
  else reg_alloc<chunk_regs(D, VP)>();
  if (helper && !producer) return;
  bool live = true;                            // false after a wait ran out: no further waits
  auto wait_for = [&](uint32_t bar, uint32_t parity) {
    if (live && !mbar_wait_bounded(bar, parity)) {
      arcb_set_error(a.err, ARCB_DEV_WAIT_TIMEOUT_TMA);
      live = false;
    }
  };
  // rows behind the segment's end are other rows' data (or zeros): finite, and weighted by zero
  auto load_tiles = [&](int c) {
    const uint32_t st = base + (c & 1) * C::STAGE, full = bars + 8 * (c & 1);
    const int y = row0 + c * L;
    mbar_expect_tx(full, 2 * C::QB + C::VB);
#pragma unroll
    for (int b = 0; b < D / 64; ++b) {
      tma_load_2d(st + b * (L * 128), &tmap, a.off_q + h * D + b * 64, y, full);
      tma_load_2d(st + C::Q_TILE + b * (L * 128), &tmap, a.off_k + h * D + b * 64, y, full);
    }
#pragma unroll
    for (int b = 0; b < VP / 64; ++b) tma_load_2d(st + C::Q_TILE + C::QB + b * (L * 128), &tmap, a.off_v + h * VP + b * 64, y, full);
  };
  // gates of chunk c from the stabiliser before it; returns the stabiliser after it.  Lane: tokens 2 lane, 2 lane + 1
  auto make_gates = [&](int c, float m0) -> float {
    float* fg = f_gate + (c & 1) * C::GATE_FLOATS;
    float gi[2], gf[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = c * L + 2 * lane + e;
      const bool ok = t < rows;
      const float* gr = a.gates + (size_t)(row0 + (ok ? t : 0)) * 2 * a.H + h;
      gi[e] = ok ? gr[0] : 0.f;
      gf[e] = ok ? gr[a.H] : 0.f;
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool ok = c * L + 2 * lane + e < rows;
      gi[e] = ok ? gate_log(gi[e], a.gate_cap, false) : -INFINITY;
      gf[e] = ok ? gate_log(gf[e], a.gate_cap, true) : 0.f;
    }
    float run = gf[0] + gf[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += x;
    }
    const float F1 = run, F0 = run - gf[1];
    const float c0 = gi[0] - F0, c1 = gi[1] - F1;
    float mx = fmaxf(c0, c1);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, mx, o);
      if (lane >= o) mx = fmaxf(mx, x);
    }
    float before = __shfl_up_sync(0xffffffffu, mx, 1);
    if (lane == 0) before = -INFINITY;
    const float M0 = fmaxf(m0, fmaxf(before, c0)), M1 = fmaxf(m0, mx);
    const float ML = __shfl_sync(0xffffffffu, M1, 31);
    const float FL = __shfl_sync(0xffffffffu, F1, 31);
    const float2 out[5] = {make_float2(c0 * LOG2E, c1 * LOG2E), make_float2(M0 * LOG2E, M1 * LOG2E),
                           make_float2(expf(c0 - ML), expf(c1 - ML)), make_float2(expf(m0 - M0), expf(m0 - M1)),
                           make_float2(expf(-(F0 + M0)), expf(-(F1 + M1)))};
#pragma unroll
    for (int i = 0; i < 5; ++i) *reinterpret_cast<float2*>(fg + i * L + 2 * lane) = out[i];
    if (lane == 0) { fg[5 * L] = expf(m0 - ML); fg[5 * L + 1] = FL + ML; }
    return FL + ML;
  };
  auto chunk_barrier = [&]() { named_bar_sync(1, C::NB); };

  if (producer) {
    if (lane == 0) load_tiles(0);
    m = make_gates(0, m);
    chunk_barrier();
    for (int c = 0; c < n_chunks; ++c) {
      if (c + 1 < n_chunks) {
        if (lane == 0) {
          fence_proxy_async_smem();   // the stage's last readers are behind a barrier
          load_tiles(c + 1);
        }
        m = make_gates(c + 1, m);
      }
      chunk_barrier();                // the queries have been read
      if (lane == 0) {
        fence_proxy_async_smem();
        mbar_expect_tx(bars + 16, C::VB);
#pragma unroll
        for (int b = 0; b < VP / 64; ++b)
          tma_load_2d(base + (c & 1) * C::STAGE + b * (L * 128), &tmap, a.off_g + h * VP + b * 64, row0 + c * L, bars + 16);
      }
      chunk_barrier();
      chunk_barrier();
    }
    if (lane == 0) *mg = m;
    return;
  }

  float S[D / 8][4];                         // tile nt: (v_lo, d), (v_lo, d + 1), (v_lo + 8, d), (v_lo + 8, d + 1), d = 8 nt + 2 t4
#pragma unroll
  for (int nt = 0; nt < D / 8; ++nt) {
    const int d = nt * 8 + 2 * t4;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int dd = d + (e & 1), v = v_lo + (e >> 1) * 8;
      S[nt][e] = (!fresh && dd < a.dim) ? Sg[(size_t)dd * VP + v] : 0.f;
    }
  }
  const int rt_s = warp & 3, kh = warp >> 2;  // score block of this warp: token rows, key half
  const float inv_v = 1.f / (float)a.vdim;
  float2 gain[2];
#pragma unroll
  for (int nt = 0; nt < 2; ++nt)
    gain[nt] = __ldg(reinterpret_cast<const float2*>(a.norm_w + (size_t)h * VP + warp * 16 + nt * 8 + 2 * t4));
  uint16_t* out = reinterpret_cast<uint16_t*>(a.out) + ((size_t)row0 * a.H + h) * VP + warp * 16 + 2 * t4;
  chunk_barrier();

  for (int c = 0; c < n_chunks; ++c) {
    const int buf = c & 1, t0 = c * L;
    const int n_tok = min(L, rows - t0);
    const float* fg = f_gate + buf * C::GATE_FLOATS;
    const float* f_c = fg;            // c_s log2 e
    const float* f_M = fg + L;        // M_t log2 e
    const float* f_w = fg + 2 * L;    // exp(c_s - M_L)
    const float* f_row = fg + 3 * L;  // exp(m - M_t)
    const float* f_em = fg + 4 * L;   // exp(-m_t)
    const float keep = fg[5 * L];     // exp(m - M_L)
    wait_for(bars + 8 * buf, (c >> 1) & 1);
    const uint32_t q_s = base + buf * C::STAGE, k_s = q_s + C::Q_TILE, v_s = k_s + C::QB;

    // ---- n . q of the carried state: NC / L threads a row ----
    {
      constexpr int TPR = NC / L;
      const int r = tid / TPR, part = tid % TPR;
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < D / 8 / TPR; ++i) {
        const int ch = part + i * TPR;
        const uint4 q4 = *reinterpret_cast<const uint4*>(bp + buf * C::STAGE + tile_off(r, ch));
        const uint32_t qw[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 q2 = unpack2_act(qw[e], F16 ? 1 : 0);
          const float2 n2 = *reinterpret_cast<const float2*>(f_n + ch * 8 + 2 * e);
          s = fmaf(q2.x, n2.x, s);
          s = fmaf(q2.y, n2.y, s);
        }
      }
#pragma unroll
      for (int o = 1; o < TPR; o <<= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (part == 0) f_qn[r] = s;
    }
    // ---- decay-weighted scores of this warp's block: 16 tokens x L / KH keys ----
    {
      constexpr int NTILES = L / 8 / KH;
      float sc[NTILES][4];
#pragma unroll
      for (int i = 0; i < NTILES; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[i][e] = 0.f;
      const bool below = kh * (L / KH) <= rt_s * 16 + 15;     // some key of the block is visible
      if (below) {
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {
          uint32_t qa[4];
          ldsm4(q_s + tile_off(rt_s * 16 + (lane & 15), ks * 2 + (lane >> 4)), qa);
#pragma unroll
          for (int np = 0; np < NTILES / 2; ++np) {
            uint32_t kb[4];
            ldsm4(k_s + tile_off(kh * (L / KH) + np * 16 + (lane & 7) + (lane >> 4) * 8, ks * 2 + ((lane >> 3) & 1)), kb);
            mma16816<F16>(sc[2 * np], qa, kb[0], kb[1]);
            mma16816<F16>(sc[2 * np + 1], qa, kb[2], kb[3]);
          }
        }
      }
      const int r_lo = rt_s * 16 + g;
      const float M_lo = f_M[r_lo], M_hi = f_M[r_lo + 8];
      float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
      for (int i = 0; i < NTILES; ++i) {
        const int s0 = kh * (L / KH) + i * 8 + 2 * t4;
        const float2 cs = *reinterpret_cast<const float2*>(f_c + s0);
        const float p00 = s0 <= r_lo ? sc[i][0] * ex2_approx(cs.x - M_lo) : 0.f;
        const float p01 = s0 + 1 <= r_lo ? sc[i][1] * ex2_approx(cs.y - M_lo) : 0.f;
        const float p10 = s0 <= r_lo + 8 ? sc[i][2] * ex2_approx(cs.x - M_hi) : 0.f;
        const float p11 = s0 + 1 <= r_lo + 8 ? sc[i][3] * ex2_approx(cs.y - M_hi) : 0.f;
        sum_lo += p00 + p01;
        sum_hi += p10 + p11;
        const int ch = (s0 >> 3), in = (s0 & 7) * 2;
        *reinterpret_cast<uint32_t*>(bp + 2 * C::STAGE + tile_off(r_lo, ch) + in) = pack2_act(p00, p01, F16 ? 1 : 0);
        *reinterpret_cast<uint32_t*>(bp + 2 * C::STAGE + tile_off(r_lo + 8, ch) + in) = pack2_act(p10, p11, F16 ? 1 : 0);
      }
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        sum_lo += __shfl_xor_sync(0xffffffffu, sum_lo, o);
        sum_hi += __shfl_xor_sync(0xffffffffu, sum_hi, o);
      }
      if (t4 == 0) { f_sum[kh * L + r_lo] = sum_lo; f_sum[kh * L + r_lo + 8] = sum_hi; }
    }
    // ---- carried state: acc = Q S for all tokens and this warp's 16 value columns ----
    float acc[L / 16][2][4];
#pragma unroll
    for (int rt = 0; rt < L / 16; ++rt)
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[rt][nt][e] = 0.f;
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks) {
      uint32_t bh[4], bl[4];
      split2<F16>(S[2 * ks][0] * S_SCALE, S[2 * ks][1] * S_SCALE, bh[0], bl[0]);
      split2<F16>(S[2 * ks + 1][0] * S_SCALE, S[2 * ks + 1][1] * S_SCALE, bh[1], bl[1]);
      split2<F16>(S[2 * ks][2] * S_SCALE, S[2 * ks][3] * S_SCALE, bh[2], bl[2]);
      split2<F16>(S[2 * ks + 1][2] * S_SCALE, S[2 * ks + 1][3] * S_SCALE, bh[3], bl[3]);
      uint32_t qa[L / 16][4];
#pragma unroll
      for (int rt = 0; rt < L / 16; ++rt) {
        ldsm4(q_s + tile_off(rt * 16 + (lane & 15), ks * 2 + (lane >> 4)), qa[rt]);
        mma16816<F16>(acc[rt][0], qa[rt], bh[0], bh[1]);
        mma16816<F16>(acc[rt][1], qa[rt], bh[2], bh[3]);
      }
#pragma unroll
      for (int rt = 0; rt < L / 16; ++rt) {    // the remainders, clear of the products they follow
        mma16816<F16>(acc[rt][0], qa[rt], bl[0], bl[1]);
        mma16816<F16>(acc[rt][1], qa[rt], bl[2], bl[3]);
      }
    }
    chunk_barrier();     // P, its sums and n . q are complete
    // ---- add the chunk's own part, normalise ----
#pragma unroll
    for (int rt = 0; rt < L / 16; ++rt) {
      const int r_lo = rt * 16 + g, r_hi = r_lo + 8;
      const float e_lo = f_row[r_lo], e_hi = f_row[r_hi];
      const float u_lo = e_lo * (1.f / S_SCALE), u_hi = e_hi * (1.f / S_SCALE);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        acc[rt][nt][0] *= u_lo; acc[rt][nt][1] *= u_lo;
        acc[rt][nt][2] *= u_hi; acc[rt][nt][3] *= u_hi;
      }
#pragma unroll
      for (int ks = 0; ks <= rt; ++ks) {       // keys beyond the row tile are hidden
        uint32_t pa[4], vb[4];
        ldsm4(p_smem + tile_off(rt * 16 + (lane & 15), ks * 2 + (lane >> 4)), pa);
        ldsm4_t(v_s + tile_off(ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, warp * 2 + (lane >> 4)), vb);
        mma16816<F16>(acc[rt][0], pa, vb[0], vb[1]);
        mma16816<F16>(acc[rt][1], pa, vb[2], vb[3]);
      }
      float nq_lo = e_lo * f_qn[r_lo] + f_sum[r_lo], nq_hi = e_hi * f_qn[r_hi] + f_sum[r_hi];
      if (KH == 2) { nq_lo += f_sum[L + r_lo]; nq_hi += f_sum[L + r_hi]; }
      const float d_lo = __fdividef(1.f, fmaxf(fabsf(nq_lo), f_em[r_lo]) + 1e-6f), d_hi = __fdividef(1.f, fmaxf(fabsf(nq_hi), f_em[r_hi]) + 1e-6f);
      float s_lo = 0.f, s_hi = 0.f;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        acc[rt][nt][0] *= d_lo; acc[rt][nt][1] *= d_lo;
        acc[rt][nt][2] *= d_hi; acc[rt][nt][3] *= d_hi;
        s_lo += acc[rt][nt][0] * acc[rt][nt][0] + acc[rt][nt][1] * acc[rt][nt][1];
        s_hi += acc[rt][nt][2] * acc[rt][nt][2] + acc[rt][nt][3] * acc[rt][nt][3];
      }
#pragma unroll
      for (int o = 1; o < 4; o <<= 1) {
        s_lo += __shfl_xor_sync(0xffffffffu, s_lo, o);
        s_hi += __shfl_xor_sync(0xffffffffu, s_hi, o);
      }
      if (t4 == 0) { f_ss[warp * L + r_lo] = s_lo; f_ss[warp * L + r_hi] = s_hi; }
    }
    // ---- state: S^T <- exp(m - M_L) S^T + (V w)^T K ----
    {
#pragma unroll
      for (int nt = 0; nt < D / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[nt][e] *= keep;
#pragma unroll
      for (int ks = 0; ks < L / 16; ++ks) {
        uint32_t va[4], vh[4], vl[4];
        ldsm4_t(v_s + tile_off(ks * 16 + (lane & 7) + (lane >> 4) * 8, warp * 2 + ((lane >> 3) & 1)), va);
        const float2 w0 = *reinterpret_cast<const float2*>(f_w + ks * 16 + 2 * t4), w1 = *reinterpret_cast<const float2*>(f_w + ks * 16 + 8 + 2 * t4);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 v2 = unpack2_act(va[e], F16 ? 1 : 0);
          const float2 w = e < 2 ? w0 : w1;
          split2<F16>(v2.x * w.x, v2.y * w.y, vh[e], vl[e]);
        }
#pragma unroll
        for (int np = 0; np < D / 16; np += 2) {
          uint32_t kb[2][4];
#pragma unroll
          for (int x = 0; x < 2; ++x)
            ldsm4_t(k_s + tile_off(ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, (np + x) * 2 + (lane >> 4)), kb[x]);
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            mma16816<F16>(S[2 * (np + x)], vh, kb[x][0], kb[x][1]);
            mma16816<F16>(S[2 * (np + x) + 1], vh, kb[x][2], kb[x][3]);
          }
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            mma16816<F16>(S[2 * (np + x)], vl, kb[x][0], kb[x][1]);
            mma16816<F16>(S[2 * (np + x) + 1], vl, kb[x][2], kb[x][3]);
          }
        }
      }
    }
    // ---- n: column sums of the weighted keys, in NP groups of tokens ----
    constexpr int NP = 2 * NC / D > 4 ? 4 : 2 * NC / D;
    for (int i = tid; i < NP * (D / 2); i += NC) {
      const int dp = i % (D / 2), part = i / (D / 2);
      float s0 = 0.f, s1 = 0.f;
#pragma unroll 8
      for (int t = 0; t < L / NP; ++t) {
        const int r = part * (L / NP) + t;
        const float2 k2 = unpack2_act(*reinterpret_cast<const uint32_t*>(bp + buf * C::STAGE + C::Q_TILE + tile_off(r, dp >> 2) + (dp & 3) * 4), F16 ? 1 : 0);
        s0 = fmaf(f_w[r], k2.x, s0);
        s1 = fmaf(f_w[r], k2.y, s1);
      }
      *reinterpret_cast<float2*>(f_np + part * D + 2 * dp) = make_float2(s0, s1);
    }
    chunk_barrier();     // squares and n partials are complete
    for (int d = tid; d < D; d += NC) {
      float s = keep * f_n[d];
#pragma unroll
      for (int i = 0; i < NP; ++i) s += f_np[i * D + d];
      f_n[d] = s;
    }
    wait_for(bars + 16, c & 1);     // the output gates
    // ---- head norm, gain, output gate ----
    float inv[L / 16][2];
#pragma unroll
    for (int rt = 0; rt < L / 16; ++rt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float ss = 0.f;
#pragma unroll
        for (int w = 0; w < NW; ++w) ss += f_ss[w * L + rt * 16 + g + e * 8];
        inv[rt][e] = rsqrtf(ss * inv_v + a.eps);
      }
#pragma unroll
    for (int rt = 0; rt < L / 16; ++rt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = rt * 16 + g + e * 8;
        uint16_t* dst = out + (size_t)(t0 + r) * (a.H * VP);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const float2 gt = unpack2_act(*reinterpret_cast<const uint32_t*>(bp + buf * C::STAGE + tile_off(r, warp * 2 + nt) + 4 * t4), F16 ? 1 : 0);
          const uint32_t o = pack2_act(acc[rt][nt][2 * e] * inv[rt][e] * gain[nt].x * gt.x,
                                       acc[rt][nt][2 * e + 1] * inv[rt][e] * gain[nt].y * gt.y, F16 ? 1 : 0);
          if (r < n_tok) *reinterpret_cast<uint32_t*>(dst + nt * 8) = o;
        }
      }
    chunk_barrier();     // n is updated; the tiles and the gates' buffer are free
  }
#pragma unroll
  for (int nt = 0; nt < D / 8; ++nt) {
    const int d = nt * 8 + 2 * t4;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int dd = d + (e & 1), v = v_lo + (e >> 1) * 8;
      if (dd < a.dim) Sg[(size_t)dd * VP + v] = S[nt][e];
    }
  }
  for (int d = tid; d < a.dim; d += NC) ng[d] = f_n[d];
}

// the re-division of registers must fit what the kernel is launched with, or its increase would wait for good
template <int D, int VP, bool F16>
cudaError_t check_regs() {
  using C = ChunkCfg<D, VP>;
  cudaFuncAttributes at;
  const cudaError_t e = cudaFuncGetAttributes(&at, mlstm_chunk_kernel<F16, D, VP>);
  if (e != cudaSuccess) return e;
  return at.numRegs * C::NT >= 24 * 128 + chunk_regs(D, VP) * C::NC ? cudaSuccess : cudaErrorLaunchOutOfResources;
}

template <int D, int VP>
cudaError_t set_attr() {
  cudaError_t c = check_regs<D, VP, true>();
  if (c == cudaSuccess) c = check_regs<D, VP, false>();
  if (c != cudaSuccess) return c;
  cudaError_t e = cudaFuncSetAttribute(mlstm_chunk_kernel<true, D, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, ChunkCfg<D, VP>::SMEM);
  if (e != cudaSuccess) return e;
  return cudaFuncSetAttribute(mlstm_chunk_kernel<false, D, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, ChunkCfg<D, VP>::SMEM);
}

template <int D, int VP>
cudaError_t launch_chunk(const CUtensorMap& tm, const MlstmArgs& a, cudaStream_t stream) {
  using C = ChunkCfg<D, VP>;
  const dim3 grid(a.H, a.n_segs);
  return a.fmt == 1 ? arcb_launch(mlstm_chunk_kernel<true, D, VP>, grid, dim3(C::NT), C::SMEM, stream, tm, a)
                    : arcb_launch(mlstm_chunk_kernel<false, D, VP>, grid, dim3(C::NT), C::SMEM, stream, tm, a);
}

}  // namespace

bool arcb_mlstm_chunk_supported(int dimp, int vdimp, int fmt) { return fmt != 2 && dimp <= 128 && vdimp <= 128; }

int arcb_mlstm_chunk_init() {
  cudaError_t e;
  if ((e = set_attr<64, 64>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<64, 128>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<128, 64>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<128, 128>()) != cudaSuccess) return (int)e;
  return 0;
}

int arcb_launch_mlstm_chunk(const MlstmArgs& a, cudaStream_t stream) {
  if (a.n_segs <= 0) return 0;
  if (a.n_segs > 65535 || !a.seg_seq || a.n_rows <= 0) return -1;
  CUtensorMap tm;
  const int r = arcb_make_tmap_2d_16b(&tm, a.proj, (uint64_t)a.n_rows, (uint64_t)a.pitch, L, 64, a.fmt);
  if (r) return 1000 + r;
  cudaError_t e = cudaErrorInvalidValue;
  switch (a.dimp * 1000 + a.vdimp) {
    case 64064: e = launch_chunk<64, 64>(tm, a, stream); break;
    case 64128: e = launch_chunk<64, 128>(tm, a, stream); break;
    case 128064: e = launch_chunk<128, 64>(tm, a, stream); break;
    case 128128: e = launch_chunk<128, 128>(tm, a, stream); break;
  }
  arcb_count_launch(1);
  return (int)e;
}
