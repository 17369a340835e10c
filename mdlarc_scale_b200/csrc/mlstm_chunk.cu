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
// Tiles arrive by cp.async, the next chunk's while this one is computed.  The products are small (64 rows) and
// the launch is bound by reading q, k, v and the gates, so warp-level MMA is enough to stay near that bound.
#include "launch.cuh"
#include "mlstm.cuh"
#include "ptx_sm100.cuh"

using namespace sm100;

namespace {

constexpr int L = 64;      // tokens per chunk

// CTAs per SM the register budget is set for (in units of 256 threads)
#ifndef ARCB_MLSTM_CHUNK_WIDE_CTAS
#define ARCB_MLSTM_CHUNK_WIDE_CTAS 2
#endif
__host__ __device__ constexpr int chunk_ctas(int d, int nt) { return (d == 128 ? ARCB_MLSTM_CHUNK_WIDE_CTAS : 2) * 256 / nt; }

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

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
// (x, y) as a packed pair and the packed pair of what the rounding left over
template <bool F16>
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack2_act(x, y, F16 ? 1 : 0);
  const float2 h = unpack2_act(hi, F16 ? 1 : 0);
  lo = pack2_act(x - h.x, y - h.y, F16 ? 1 : 0);
}

// byte offset of 16-byte chunk `ch` of row `row` in a tile of COLS 16-bit columns, chunks XOR-swizzled by row
template <int COLS>
__device__ __forceinline__ uint32_t tile_off(int row, int ch) {
  return (uint32_t)(row * (COLS * 2) + ((ch ^ (row & 7)) << 4));
}

template <int D, int VP>
struct ChunkCfg {
  static constexpr int NW = VP / 16;         // warps
  static constexpr int NT = NW * 32;
  static constexpr int QB = L * D * 2, VB = L * VP * 2;
  static constexpr int STAGE = 2 * QB + VB;  // q, k, v
  static constexpr int PB = L * L * 2;
  // stages | P | c, M, F, w, row factor, exp(-m_t), n.q, score sums [2][L] | n | n partials | squares [NW][L]
  static constexpr int FLOATS = 9 * L + D + 2 * D + NW * L + 8;
  static constexpr int SMEM = 2 * STAGE + PB + FLOATS * 4 + 128;
};

template <bool F16, int D, int VP>
__global__ void __launch_bounds__(ChunkCfg<D, VP>::NT, chunk_ctas(D, ChunkCfg<D, VP>::NT))
mlstm_chunk_kernel(MlstmArgs a) {
  using C = ChunkCfg<D, VP>;
  constexpr int NW = C::NW, NT = C::NT;
  constexpr int KH = NW / 4;                 // key halves of the score blocks
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw = smem_u32(smem_raw);
  const uint32_t base = (raw + 127u) & ~127u;
  uint8_t* bp = smem_raw + (base - raw);
  const uint32_t p_smem = base + 2 * C::STAGE;
  float* f_c = reinterpret_cast<float*>(bp + 2 * C::STAGE + C::PB);
  float* f_M = f_c + L;
  float* f_w = f_M + L;          // exp(c_s - M_L)
  float* f_row = f_w + L;        // exp(m - M_t)
  float* f_em = f_row + L;       // exp(-m_t)
  float* f_qn = f_em + L;        // n . q_t of the carried state
  float* f_sum = f_qn + L;       // [KH <= 2][L] score sums
  float* f_n = f_sum + 2 * L;    // [D]
  float* f_np = f_n + D;         // [2][D]
  float* f_ss = f_np + 2 * D;    // [NW][L]
  float* f_misc = f_ss + NW * L; // [0] exp(m - M_L), [1] m at the chunk's end

  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
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
  for (int d = tid; d < D; d += NT) f_n[d] = (!fresh && d < a.dim) ? ng[d] : 0.f;
  float m = fresh ? 0.f : *mg;

  const uint16_t* proj = reinterpret_cast<const uint16_t*>(a.proj);
  auto load_tiles = [&](int c, int buf) {
    const uint32_t st = base + buf * C::STAGE;
    const int t0 = c * L;
    for (int i = tid; i < L * (D / 8); i += NT) {
      const int r = i / (D / 8), ch = i % (D / 8);
      const bool ok = t0 + r < rows;
      const uint16_t* src = proj + (size_t)(row0 + (ok ? t0 + r : 0)) * a.pitch + (size_t)h * D + ch * 8;
      cp_async16(st + tile_off<D>(r, ch), src + a.off_q, ok);
      cp_async16(st + C::QB + tile_off<D>(r, ch), src + a.off_k, ok);
    }
    for (int i = tid; i < L * (VP / 8); i += NT) {
      const int r = i / (VP / 8), ch = i % (VP / 8);
      const bool ok = t0 + r < rows;
      cp_async16(st + 2 * C::QB + tile_off<VP>(r, ch), proj + (size_t)(row0 + (ok ? t0 + r : 0)) * a.pitch + a.off_v + (size_t)h * VP + ch * 8, ok);
    }
    cp_async_commit();
  };
  const int n_chunks = (rows + L - 1) / L;
  load_tiles(0, 0);
  const int rt_s = warp & 3, kh = warp >> 2;  // score block of this warp: token rows, key half
  const float inv_v = 1.f / (float)a.vdim;

  for (int c = 0; c < n_chunks; ++c) {
    const int buf = c & 1, t0 = c * L;
    const int n_tok = min(L, rows - t0);
    if (c + 1 < n_chunks) load_tiles(c + 1, buf ^ 1);
    if (warp == 0) {
      // gates of the chunk: lane owns tokens 2 lane, 2 lane + 1
      float gi[2], gf[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = 2 * lane + e;
        const bool ok = t < n_tok;
        const float* gr = a.gates + (size_t)(row0 + t0 + (ok ? t : 0)) * 2 * a.H + h;
        gi[e] = ok ? gate_log(gr[0], a.gate_cap, false) : -INFINITY;
        gf[e] = ok ? gate_log(gr[a.H], a.gate_cap, true) : 0.f;
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
      const float M0 = fmaxf(m, fmaxf(before, c0)), M1 = fmaxf(m, mx);
      const float ML = __shfl_sync(0xffffffffu, M1, 31);
      const float FL = __shfl_sync(0xffffffffu, F1, 31);
      f_c[2 * lane] = c0; f_c[2 * lane + 1] = c1;
      f_M[2 * lane] = M0; f_M[2 * lane + 1] = M1;
      f_w[2 * lane] = expf(c0 - ML); f_w[2 * lane + 1] = expf(c1 - ML);
      f_row[2 * lane] = expf(m - M0); f_row[2 * lane + 1] = expf(m - M1);
      f_em[2 * lane] = expf(-(F0 + M0)); f_em[2 * lane + 1] = expf(-(F1 + M1));
      if (lane == 0) { f_misc[0] = expf(m - ML); f_misc[1] = FL + ML; }
    }
    if (c + 1 < n_chunks) cp_async_wait<1>(); else cp_async_wait<0>();
    __syncthreads();
    const uint32_t q_s = base + buf * C::STAGE, k_s = q_s + C::QB, v_s = q_s + 2 * C::QB;

    // ---- n . q of the carried state: NT / L threads a row ----
    {
      constexpr int TPR = NT / L;
      const int r = tid / TPR, part = tid % TPR;
      float s = 0.f;
#pragma unroll
      for (int i = 0; i < D / 8 / TPR; ++i) {
        const int ch = part + i * TPR;
        const uint4 q4 = *reinterpret_cast<const uint4*>(bp + buf * C::STAGE + tile_off<D>(r, ch));
        const uint32_t qw[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 q2 = unpack2_act(qw[e], F16 ? 1 : 0);
          s = fmaf(q2.x, f_n[ch * 8 + 2 * e], s);
          s = fmaf(q2.y, f_n[ch * 8 + 2 * e + 1], s);
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
          ldsm4(q_s + tile_off<D>(rt_s * 16 + (lane & 15), ks * 2 + (lane >> 4)), qa);
#pragma unroll
          for (int np = 0; np < NTILES / 2; ++np) {
            uint32_t kb[4];
            ldsm4(k_s + tile_off<D>(kh * (L / KH) + np * 16 + (lane & 7) + (lane >> 4) * 8, ks * 2 + ((lane >> 3) & 1)), kb);
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
        const float c0 = f_c[s0], c1 = f_c[s0 + 1];
        const float p00 = s0 <= r_lo ? sc[i][0] * __expf(c0 - M_lo) : 0.f;
        const float p01 = s0 + 1 <= r_lo ? sc[i][1] * __expf(c1 - M_lo) : 0.f;
        const float p10 = s0 <= r_lo + 8 ? sc[i][2] * __expf(c0 - M_hi) : 0.f;
        const float p11 = s0 + 1 <= r_lo + 8 ? sc[i][3] * __expf(c1 - M_hi) : 0.f;
        sum_lo += p00 + p01;
        sum_hi += p10 + p11;
        const int ch = (s0 >> 3), in = (s0 & 7) * 2;
        *reinterpret_cast<uint32_t*>(bp + 2 * C::STAGE + tile_off<L>(r_lo, ch) + in) = pack2_act(p00, p01, F16 ? 1 : 0);
        *reinterpret_cast<uint32_t*>(bp + 2 * C::STAGE + tile_off<L>(r_lo + 8, ch) + in) = pack2_act(p10, p11, F16 ? 1 : 0);
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
      split2<F16>(S[2 * ks][0], S[2 * ks][1], bh[0], bl[0]);
      split2<F16>(S[2 * ks + 1][0], S[2 * ks + 1][1], bh[1], bl[1]);
      split2<F16>(S[2 * ks][2], S[2 * ks][3], bh[2], bl[2]);
      split2<F16>(S[2 * ks + 1][2], S[2 * ks + 1][3], bh[3], bl[3]);
#pragma unroll
      for (int rt = 0; rt < L / 16; ++rt) {
        uint32_t qa[4];
        ldsm4(q_s + tile_off<D>(rt * 16 + (lane & 15), ks * 2 + (lane >> 4)), qa);
        mma16816<F16>(acc[rt][0], qa, bh[0], bh[1]);
        mma16816<F16>(acc[rt][0], qa, bl[0], bl[1]);
        mma16816<F16>(acc[rt][1], qa, bh[2], bh[3]);
        mma16816<F16>(acc[rt][1], qa, bl[2], bl[3]);
      }
    }
    __syncthreads();     // P, its sums and n . q are complete
    // ---- add the chunk's own part, normalise ----
#pragma unroll
    for (int rt = 0; rt < L / 16; ++rt) {
      const int r_lo = rt * 16 + g, r_hi = r_lo + 8;
      const float e_lo = f_row[r_lo], e_hi = f_row[r_hi];
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        acc[rt][nt][0] *= e_lo; acc[rt][nt][1] *= e_lo;
        acc[rt][nt][2] *= e_hi; acc[rt][nt][3] *= e_hi;
      }
#pragma unroll
      for (int ks = 0; ks <= rt; ++ks) {       // keys beyond the row tile are hidden
        uint32_t pa[4], vb[4];
        ldsm4(p_smem + tile_off<L>(rt * 16 + (lane & 15), ks * 2 + (lane >> 4)), pa);
        ldsm4_t(v_s + tile_off<VP>(ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, warp * 2 + (lane >> 4)), vb);
        mma16816<F16>(acc[rt][0], pa, vb[0], vb[1]);
        mma16816<F16>(acc[rt][1], pa, vb[2], vb[3]);
      }
      float nq_lo = e_lo * f_qn[r_lo] + f_sum[r_lo], nq_hi = e_hi * f_qn[r_hi] + f_sum[r_hi];
      if (KH == 2) { nq_lo += f_sum[L + r_lo]; nq_hi += f_sum[L + r_hi]; }
      const float d_lo = 1.f / (fmaxf(fabsf(nq_lo), f_em[r_lo]) + 1e-6f), d_hi = 1.f / (fmaxf(fabsf(nq_hi), f_em[r_hi]) + 1e-6f);
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
      const float keep = f_misc[0];
#pragma unroll
      for (int nt = 0; nt < D / 8; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[nt][e] *= keep;
#pragma unroll
      for (int ks = 0; ks < L / 16; ++ks) {
        uint32_t va[4], vh[4], vl[4];
        ldsm4_t(v_s + tile_off<VP>(ks * 16 + (lane & 7) + (lane >> 4) * 8, warp * 2 + ((lane >> 3) & 1)), va);
        const float2 w0 = *reinterpret_cast<const float2*>(f_w + ks * 16 + 2 * t4), w1 = *reinterpret_cast<const float2*>(f_w + ks * 16 + 8 + 2 * t4);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 v2 = unpack2_act(va[e], F16 ? 1 : 0);
          const float2 w = e < 2 ? w0 : w1;
          split2<F16>(v2.x * w.x, v2.y * w.y, vh[e], vl[e]);
        }
#pragma unroll
        for (int np = 0; np < D / 16; ++np) {
          uint32_t kb[4];
          ldsm4_t(k_s + tile_off<D>(ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8, np * 2 + (lane >> 4)), kb);
          mma16816<F16>(S[2 * np], vh, kb[0], kb[1]);
          mma16816<F16>(S[2 * np], vl, kb[0], kb[1]);
          mma16816<F16>(S[2 * np + 1], vh, kb[2], kb[3]);
          mma16816<F16>(S[2 * np + 1], vl, kb[2], kb[3]);
        }
      }
    }
    // ---- n: column sums of the weighted keys, two token halves ----
    for (int i = tid; i < 2 * (D / 2); i += NT) {
      const int dp = i % (D / 2), part = i / (D / 2);
      float s0 = 0.f, s1 = 0.f;
#pragma unroll 8
      for (int t = 0; t < L / 2; ++t) {
        const int r = part * (L / 2) + t;
        const float2 k2 = unpack2_act(*reinterpret_cast<const uint32_t*>(bp + buf * C::STAGE + C::QB + tile_off<D>(r, dp >> 2) + (dp & 3) * 4), F16 ? 1 : 0);
        s0 = fmaf(f_w[r], k2.x, s0);
        s1 = fmaf(f_w[r], k2.y, s1);
      }
      f_np[part * D + 2 * dp] = s0;
      f_np[part * D + 2 * dp + 1] = s1;
    }
    __syncthreads();     // squares and n partials are complete; the tiles are free
    for (int d = tid; d < D; d += NT) f_n[d] = f_misc[0] * f_n[d] + (f_np[d] + f_np[D + d]);
    m = f_misc[1];
    // ---- head norm, gain, output gate ----
#pragma unroll
    for (int rt = 0; rt < L / 16; ++rt)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = rt * 16 + g + e * 8;
        if (r >= n_tok) continue;
        float ss = 0.f;
#pragma unroll
        for (int w = 0; w < NW; ++w) ss += f_ss[w * L + r];
        const float inv = 1.f / sqrtf(ss * inv_v + a.eps);
        const size_t row = (size_t)row0 + t0 + r;
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          const int v = warp * 16 + nt * 8 + 2 * t4;
          const float2 gt = unpack2_act(__ldg(reinterpret_cast<const uint32_t*>(proj + row * a.pitch + a.off_g + (size_t)h * VP + v)), F16 ? 1 : 0);
          const float2 nw = __ldg(reinterpret_cast<const float2*>(a.norm_w + (size_t)h * VP + v));
          const uint32_t o = pack2_act(acc[rt][nt][2 * e] * inv * nw.x * gt.x, acc[rt][nt][2 * e + 1] * inv * nw.y * gt.y, F16 ? 1 : 0);
          *reinterpret_cast<uint32_t*>(reinterpret_cast<uint16_t*>(a.out) + (row * a.H + h) * VP + v) = o;
        }
      }
    __syncthreads();     // n is updated; the scalars may be rewritten
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
  for (int d = tid; d < a.dim; d += NT) ng[d] = f_n[d];
  if (tid == 0) *mg = m;
}

template <int D, int VP>
cudaError_t set_attr() {
  cudaError_t e = cudaFuncSetAttribute(mlstm_chunk_kernel<true, D, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, ChunkCfg<D, VP>::SMEM);
  if (e != cudaSuccess) return e;
  return cudaFuncSetAttribute(mlstm_chunk_kernel<false, D, VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, ChunkCfg<D, VP>::SMEM);
}

template <int D, int VP>
cudaError_t launch_chunk(const MlstmArgs& a, cudaStream_t stream) {
  using C = ChunkCfg<D, VP>;
  const dim3 grid(a.H, a.n_segs);
  return a.fmt == 1 ? arcb_launch(mlstm_chunk_kernel<true, D, VP>, grid, dim3(C::NT), C::SMEM, stream, a)
                    : arcb_launch(mlstm_chunk_kernel<false, D, VP>, grid, dim3(C::NT), C::SMEM, stream, a);
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
  if (a.n_segs > 65535 || !a.seg_seq) return -1;
  cudaError_t e = cudaErrorInvalidValue;
  switch (a.dimp * 1000 + a.vdimp) {
    case 64064: e = launch_chunk<64, 64>(a, stream); break;
    case 64128: e = launch_chunk<64, 128>(a, stream); break;
    case 128064: e = launch_chunk<128, 64>(a, stream); break;
    case 128128: e = launch_chunk<128, 128>(a, stream); break;
  }
  arcb_count_launch(1);
  return (int)e;
}
