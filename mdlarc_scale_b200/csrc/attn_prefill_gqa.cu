// Causal prefill attention of grouped heads on tcgen05 tensor cores with TMEM accumulators, reading keys and
// values straight from the cache (so a portion of a prompt sees what earlier portions left there).
//
// One CTA = up to 256 consecutive query rows of one sequence (two 128-row Q tiles, A and B) x one query head.
// Warps 0-3 are helpers (TMA producer, MMA issuer of A, MMA issuer of B, one idle); warps 4-11 serve tile A
// and warps 12-19 tile B, two threads per query row: thread `half` owns keys [64 half, 64 half + 64) of every
// 128-key tile and half of the output dims.  Per key tile j and Q tile x:
//   TMA        K and V tiles as 128 x 64 boxes, 128-byte swizzle, rings shared by A and B
//   MMA        S_x = Q_x K^T, fp32 in 128 TMEM columns
//   softmax_x  scores to registers; reference maximum (raised only when exceeded by 2^8, O rescaled then);
//              p = exp2(s c - m) in fp32, row sums in fp32; P rounded to the operand format and written over
//              the thread's own score columns
//   MMA        O_x += P_x V (A = P from TMEM), then at once S_x of the next tile
// Both products of a tile are issued by one thread in this order, so S(j + 1) cannot overtake the read of P(j)
// it overwrites, and its completion implies that O(j) is complete.  While one Q tile is in the tensor core the
// other tile's threads do exponentials.  A sink only joins the denominator at the end: rows are normalised by
// l 2^m + 2^(sink log2 e).  The output gate multiplies the normalised row.  Every wait is bounded.
//
// A window hides keys from below: key tiles start at the first key the block's first row sees, and tile B skips
// the tiles that lie ahead of its own first key.  With DR > 0 keys and values are those expanded from cached
// latents: the first DP key columns and the values come from the expansion scratch, the last DR key columns,
// which all heads share, from the latent cache itself.
#include <type_traits>

#include "attn_prefill_gqa.cuh"
#include "flash_common.cuh"
#include "gemm.cuh"
#include "launch.cuh"

using namespace sm100;

namespace {

constexpr int BQ = 128, BKV = 128;
constexpr int THREADS = 640;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float RESCALE_THRESHOLD = 8.f;   // log2 units
constexpr int BOX_BYTES = 128 * 64 * 2;    // one 128-row x 64-column box

template <int DP, int DR, int VP>
struct FgCfg {
  static constexpr int QB = (DP + DR) / 64;  // boxes of a query (key) row
  static constexpr int Q_BYTES = QB * BOX_BYTES;
  static constexpr int K_BYTES = Q_BYTES;
  static constexpr int V_BYTES = (VP / 64) * BOX_BYTES;
  static constexpr int AVAIL = (DR > 0 ? 224 : 208) * 1024 - 2 * Q_BYTES;
  static constexpr int FIT = AVAIL / (K_BYTES + V_BYTES);
  static constexpr int V_STAGES = FIT > 4 ? 4 : FIT;
  // one more key tile where it fits: the next tile's scores then do not wait for this tile's values
  static constexpr int K_STAGES = V_STAGES < 4 && AVAIL >= (V_STAGES + 1) * K_BYTES + V_STAGES * V_BYTES ? V_STAGES + 1 : V_STAGES;
  static_assert(V_STAGES >= 1, "a key tile and a value tile must fit");
  static constexpr int TILES = 2 * Q_BYTES + K_STAGES * K_BYTES + V_STAGES * V_BYTES;
  // DR = 0: 1 KB of alignment slack; exchange buffer and counts in static shared memory.  DR > 0 has no room for
  // either: no static shared memory (the dynamic part then starts aligned, which is checked), maxima exchanged as
  // bfloat16, denominators through the Q tile.
  static constexpr int SMEM = DR > 0 ? TILES + 320 + 2 * 2 * 2 * BQ * 2 + 64 : TILES + 1024 + 512;
  static_assert(SMEM + (DR > 0 ? 0 : 4096 + 64) <= 227 * 1024, "shared memory of one CTA");
  // S_A [0,128) S_B [128,256) O_A [256,256+VP) O_B; P_x of key half y occupies columns [64 y, 64 y + 32) of S_x
  static constexpr int TMEM_COLS = 512;
};

template <int DP, int DR, int VP, bool F16>
__global__ void __launch_bounds__(THREADS, 1)
attn_prefill_gqa_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                        const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_r,
                        AttnPrefillGqaArgs a, uint32_t idesc_qk, uint32_t idesc_pv) {
  using C = FgCfg<DP, DR, VP>;
  pdl_launch_dependents();
  pdl_wait();   // the prologue below already reads the work list from global memory
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  using XT = typename std::conditional<(DR > 0), __nv_bfloat16, float>::type;
  int* s_max_cnt;
  XT (*s_xchg)[2][2][BQ];                 // [tile parity][Q tile][half][row]
  if constexpr (DR == 0) {
    __shared__ int static_cnt[16];
    __shared__ XT static_xchg[2][2][2][BQ];
    s_max_cnt = static_cnt;
    s_xchg = static_xchg;
  } else {
    s_xchg = reinterpret_cast<XT (*)[2][2][BQ]>(smem_raw + C::TILES + 320);
    s_max_cnt = reinterpret_cast<int*>(smem_raw + C::TILES + 320 + 2 * 2 * 2 * BQ * 2);
    if (smem_u32(smem_raw) & 1023u) {
      if (threadIdx.x == 0) arcb_set_error(a.err, ARCB_DEV_BAD_INDEX);
      return;
    }
  }
  const uint32_t raw = smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - raw);
  const uint32_t q_smem = base;
  const uint32_t k_smem = base + 2 * C::Q_BYTES;
  const uint32_t v_smem = k_smem + C::K_STAGES * C::K_BYTES;
  const uint32_t bar0 = v_smem + C::V_STAGES * C::V_BYTES;
  uint8_t* bar_ptr = base_ptr + (bar0 - base);
  const uint32_t b_q = bar0, b_kfull = bar0 + 8, b_kempty = b_kfull + 8 * C::K_STAGES, b_vfull = b_kempty + 8 * C::K_STAGES,
                 b_vempty = b_vfull + 8 * C::V_STAGES, b_s = b_vempty + 8 * C::V_STAGES,
                 b_p = b_s + 16, b_o = b_p + 16, b_x = b_o + 16;     // b_x: 8 barriers, one per pair of warps of a row
  volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(bar_ptr + 256);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, blk = blockIdx.y;     // heads of a block side by side: a group's heads share its keys in L2
  const int row0 = a.qblock_row0[blk];
  const int rows = a.qblock_rows[blk];
  const int seq = a.seq[row0];
  const bool seq_ok = seq >= 0 && seq < a.n_seqs;

  const int wg = (warp >> 2) - 1;
  const int grp = wg >> 1;
  const int half = wg & 1;
  const int quarter = warp & 3;
  const int r = quarter * 32 + lane;
  int my_cnt = 0;
  // first key tile, and the first one tile B reads (rows of a block are consecutive positions)
  const int key0 = a.window > 0 && seq_ok ? max(0, a.kv_count[row0] - a.window) : 0;
  const int j0_b = a.window > 0 && seq_ok && rows > BQ ? (max(0, a.kv_count[row0 + BQ] - a.window) - key0) / BKV : 0;
  if (warp >= 4) {
    const int qr = grp * BQ + r;
    if (qr < rows && seq_ok) my_cnt = a.kv_count[row0 + qr];
    if (my_cnt > a.t_max) my_cnt = 0;
    int mx = my_cnt;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = max(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    if (lane == 0) s_max_cnt[warp - 4] = mx;
  }
  if (threadIdx.x == 0) {
    if (!seq_ok) arcb_set_error(a.err, ARCB_DEV_BAD_INDEX);
    mbar_init(b_q, 1);
    for (int s = 0; s < C::K_STAGES; ++s) {
      mbar_init(b_kfull + 8 * s, 1);
      mbar_init(b_kempty + 8 * s, 2);
    }
    for (int s = 0; s < C::V_STAGES; ++s) {
      mbar_init(b_vfull + 8 * s, 1);
      mbar_init(b_vempty + 8 * s, 2);
    }
    for (int x = 0; x < 2; ++x) {
      mbar_init(b_s + 8 * x, 1);
      mbar_init(b_p + 8 * x, 256);
      mbar_init(b_o + 8 * x, 1);
    }
    for (int i = 0; i < 8; ++i) mbar_init(b_x + 8 * i, 64);
    mbar_fence_init();
    tma_prefetch_desc(&tmap_q);
    tma_prefetch_desc(&tmap_k);
    tma_prefetch_desc(&tmap_v);
    if (DR > 0) tma_prefetch_desc(&tmap_r);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(const_cast<uint32_t*>(tmem_slot)), C::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  int cnt_a = 0, cnt_b = 0;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    cnt_a = max(cnt_a, s_max_cnt[i]);
    cnt_b = max(cnt_b, s_max_cnt[8 + i]);
  }
  const int n_a = (max(cnt_a - key0, 0) + BKV - 1) / BKV, n_b = (max(cnt_b - key0, 0) + BKV - 1) / BKV;
  const int n_tiles = max(n_a, n_b);

  if (warp < 4) {
    reg_dealloc_24();
    if (warp == 0 && lane == 0 && n_tiles > 0) {
      // ---- TMA producer ----
      const bool two = rows > BQ;
      int kv_row, k_col, v_col;
      if (DR > 0) {
        kv_row = a.kv0[blk] + key0;
        k_col = h * DP;
        v_col = a.v_col + h * VP;
      } else {
        kv_row = (seq * a.n_kv + h / (a.n_heads / a.n_kv)) * a.t_max + key0;
        k_col = v_col = 0;
      }
      const int rot_row = (seq * a.rot_panels + a.rot_panel) * a.t_max + key0;
      mbar_expect_tx(b_q, two ? 2 * C::Q_BYTES : C::Q_BYTES);
#pragma unroll
      for (int c = 0; c < C::QB; ++c) {
        tma_load_2d(q_smem + c * BOX_BYTES, &tmap_q, a.q_col + h * (DP + DR) + c * 64, row0, b_q);
        if (two) tma_load_2d(q_smem + C::Q_BYTES + c * BOX_BYTES, &tmap_q, a.q_col + h * (DP + DR) + c * 64, row0 + BQ, b_q);
      }
      for (int j = 0; j < n_tiles; ++j) {
        const int s = j % C::K_STAGES;
        if (!mbar_wait_bounded(b_kempty + 8 * s, ((j / C::K_STAGES) & 1) ^ 1)) {
          arcb_set_error(a.err, ARCB_DEV_WAIT_TIMEOUT_MMA);
          break;
        }
        const uint32_t dst = k_smem + s * C::K_BYTES;
        mbar_expect_tx(b_kfull + 8 * s, C::K_BYTES);
#pragma unroll
        for (int c = 0; c < DP / 64; ++c) tma_load_2d(dst + c * BOX_BYTES, &tmap_k, k_col + c * 64, kv_row + j * BKV, b_kfull + 8 * s);
#pragma unroll
        for (int c = 0; c < DR / 64; ++c)
          tma_load_2d(dst + (DP / 64 + c) * BOX_BYTES, &tmap_r, 0, rot_row + c * a.t_max + j * BKV, b_kfull + 8 * s);
        const int t = j % C::V_STAGES;
        if (!mbar_wait_bounded(b_vempty + 8 * t, ((j / C::V_STAGES) & 1) ^ 1)) {
          arcb_set_error(a.err, ARCB_DEV_WAIT_TIMEOUT_MMA);
          break;
        }
        mbar_expect_tx(b_vfull + 8 * t, C::V_BYTES);
#pragma unroll
        for (int c = 0; c < VP / 64; ++c)
          tma_load_2d(v_smem + t * C::V_BYTES + c * BOX_BYTES, &tmap_v, v_col + c * 64, kv_row + j * BKV, b_vfull + 8 * t);
      }
    } else if ((warp == 1 || warp == 2) && lane == 0 && n_tiles > 0) {
      // ---- MMA issuer of Q tile x ----
      const int x = warp - 1;
      const int n_x = x ? n_b : n_a;
      const int j0 = x ? j0_b : 0;
      bool ok = true;
      auto wait_or_flag = [&](uint32_t bar, uint32_t parity, int code) {
        if (ok && !mbar_wait_bounded(bar, parity)) {
          arcb_set_error(a.err, code);
          ok = false;
        }
      };
      const uint32_t t_s = tmem_base + x * 128, t_o = tmem_base + 256 + x * VP;
      auto mma_s = [&](int j) {
        const uint32_t kst = k_smem + (j % C::K_STAGES) * C::K_BYTES;
#pragma unroll
        for (int c = 0; c < C::QB; ++c) {
          const uint64_t dq = umma_desc_k_sw128(q_smem + x * C::Q_BYTES + c * BOX_BYTES);
          const uint64_t dk = umma_desc_k_sw128(kst + c * BOX_BYTES);
#pragma unroll
          for (int ks = 0; ks < 4; ++ks) umma_f16(t_s, dq + 2 * ks, dk + 2 * ks, idesc_qk, (c | ks) ? 1u : 0u);
        }
        umma_commit(b_s + 8 * x);
        umma_commit(b_kempty + 8 * (j % C::K_STAGES));
      };
      auto mma_o = [&](int j) {
        const uint32_t vst = v_smem + (j % C::V_STAGES) * C::V_BYTES;
#pragma unroll
        for (int c = 0; c < VP / 64; ++c) {
          const uint64_t dv = umma_desc_mn_sw128(vst + c * BOX_BYTES);
#pragma unroll
          for (int ks = 0; ks < BKV / 16; ++ks)
            umma_f16_ts(t_o + c * 64, t_s + (ks >> 2) * 64 + (ks & 3) * 8, dv + (uint64_t)(ks * (2048 >> 4)), idesc_pv, (j > j0 || ks) ? 1u : 0u);
        }
        umma_commit(b_vempty + 8 * (j % C::V_STAGES));
      };
      auto wait_v = [&](int j) { wait_or_flag(b_vfull + 8 * (j % C::V_STAGES), (j / C::V_STAGES) & 1, ARCB_DEV_WAIT_TIMEOUT_TMA); };
      auto wait_k = [&](int j) { wait_or_flag(b_kfull + 8 * (j % C::K_STAGES), (j / C::K_STAGES) & 1, ARCB_DEV_WAIT_TIMEOUT_TMA); };
      // stages only the other tile uses: give them back in order as they land
      auto pass = [&](int from, int to) {
        for (int j = from; ok && j < to; ++j) {
          wait_k(j);
          if (ok) mbar_arrive(b_kempty + 8 * (j % C::K_STAGES));
          wait_v(j);
          if (ok) mbar_arrive(b_vempty + 8 * (j % C::V_STAGES));
        }
      };
      if (n_x > j0) {
        pass(0, j0);
        wait_or_flag(b_q, 0, ARCB_DEV_WAIT_TIMEOUT_TMA);
        for (int j = j0; ok && j < n_x; ++j) {
          if (j > j0) {
            wait_or_flag(b_p + 8 * x, (j - 1 - j0) & 1, ARCB_DEV_WAIT_TIMEOUT_ACC);
            wait_v(j - 1);
            if (!ok) break;
            tc_fence_after();
            mma_o(j - 1);
          }
          wait_k(j);
          if (!ok) break;
          tc_fence_after();
          mma_s(j);
        }
        wait_or_flag(b_p + 8 * x, (n_x - 1 - j0) & 1, ARCB_DEV_WAIT_TIMEOUT_ACC);
        wait_v(n_x - 1);
        if (ok) {
          tc_fence_after();
          mma_o(n_x - 1);
          umma_commit(b_o + 8 * x);
        }
        pass(n_x, n_tiles);
      } else {
        pass(0, n_tiles);
      }
    }
  } else {
    reg_alloc_112();
    // ---- softmax / output threads: row r of Q tile grp, key half `half` ----
    const int n_mine = grp ? n_b : n_a, j0 = grp ? j0_b : 0;
    const int my_lo = a.window > 0 ? max(0, my_cnt - a.window) : 0;
    const uint32_t t_lane = tmem_base + ((uint32_t)(quarter * 32) << 16);
    const uint32_t t_s = t_lane + grp * 128 + half * 64;
    const uint32_t t_o = t_lane + 256 + grp * VP + half * (VP / 2);
    const uint32_t xbar = b_x + 8 * (grp * 4 + quarter);
    const float sc = a.scale * LOG2E;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    uint32_t xphase = 0;
    // hands `mine` to the row's other thread; with bfloat16 both sides go on with the rounded values
    auto exchange = [&](int slot, float& mine, float& theirs) -> bool {
      const XT sent = (XT)mine;
      mine = (float)sent;
      s_xchg[slot][grp][half][r] = sent;
      tc_fence_before();
      mbar_arrive(xbar);
      const bool good = mbar_wait_bounded(xbar, xphase);
      tc_fence_after();
      xphase ^= 1u;
      theirs = (float)s_xchg[slot][grp][half ^ 1][r];
      return good;
    };
    for (int j = j0; j < n_mine; ++j) {
      if (ok && !mbar_wait_bounded(b_s + 8 * grp, (j - j0) & 1)) {
        arcb_set_error(a.err, ARCB_DEV_WAIT_TIMEOUT_ACC);
        ok = false;
      }
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const int tile_key = key0 + j * BKV + half * 64;            // visible: [v_lo, v_hi) of the thread's 64 keys
      const int v_hi = my_cnt - tile_key, v_lo = my_lo - tile_key;
      const bool full = __all_sync(0xffffffffu, v_hi >= 64 && v_lo <= 0);
      // 32 of the thread's 64 scores; hidden keys become -inf, whose exp2 is exactly 0
      auto load_scores = [&](int c, uint32_t (&sv)[32]) {
        tmem_ld_32x32(t_s + c * 32, sv);
        tmem_wait_ld_dep(sv);
        if (!full) {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c * 32 + i >= v_hi || c * 32 + i < v_lo) sv[i] = 0xff800000u;
        }
      };
      // the scores are read twice (maximum, then exponentials): tensor memory is quicker to read again than
      // 64 registers are to hold
      float raw_mx = -INFINITY;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t sv[32];
        load_scores(c, sv);
        float mx2 = fmaxf(__uint_as_float(sv[0]), __uint_as_float(sv[1]));
#pragma unroll
        for (int i = 2; i < 32; i += 2) mx2 = max3_f32(mx2, __uint_as_float(sv[i]), __uint_as_float(sv[i + 1]));
        raw_mx = fmaxf(raw_mx, mx2);
      }
      float mine = raw_mx == -INFINITY ? -INFINITY : raw_mx * sc;
      float other;
      bool good = exchange(j & 1, mine, other);
      if (!good) arcb_set_error(a.err, ARCB_DEV_WAIT_TIMEOUT_ACC);
      ok = __all_sync(0xffffffffu, good);
      if (!ok) break;
      const float mx = fmaxf(mine, other);
      float alpha = 1.f;
      if (mx > m_ref + RESCALE_THRESHOLD) {  // also the first visible tile (m_ref = -inf)
        alpha = (m_ref == -INFINITY) ? 0.f : ex2_fast(m_ref - mx);
        m_ref = mx;
      }
      l *= alpha;
      const float m_safe = (m_ref == -INFINITY) ? 0.f : m_ref;
      const uint64_t sc2 = pack_f32x2(sc, sc), nm2 = pack_f32x2(-m_safe, -m_safe);
      if (j > j0 && __any_sync(0xffffffffu, alpha != 1.f)) {
        // S(j) was issued after P V(j - 1): O is complete and may be rescaled
#pragma unroll
        for (int c = 0; c < VP / 64; ++c) {
          uint32_t oreg[32];
          tmem_ld_32x32(t_o + c * 32, oreg);
          tmem_wait_ld_dep(oreg);
#pragma unroll
          for (int i = 0; i < 32; ++i) oreg[i] = __float_as_uint(__uint_as_float(oreg[i]) * alpha);
          tmem_st_32x32(t_o + c * 32, oreg);
        }
      }
      float ls0 = 0.f, ls1 = 0.f;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t sv[32];
        load_scores(c, sv);
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          uint32_t pr[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            float t0, t1;
            shift2_f32(sv[g * 16 + 2 * e], sv[g * 16 + 2 * e + 1], sc2, nm2, t0, t1);
            t0 = ex2_fast(t0);
            t1 = ex2_fast(t1);
            ls0 += t0;
            ls1 += t1;
            pr[e] = pack2_prob(t0, t1, F16 ? 1 : 0);
          }
          tmem_st_32x8(t_s + (c * 2 + g) * 8, pr);   // over scores this thread has already read
        }
      }
      l += ls0 + ls1;
      tmem_wait_st();
      tc_fence_before();
      mbar_arrive(b_p + 8 * grp);
    }
    float l_other = 0.f;
    if (ok && n_mine > j0) {
      bool good;
      if constexpr (DR == 0) {
        good = exchange(n_mine & 1, l, l_other);
        good = mbar_wait_bounded(b_o + 8 * grp, 0) && good;
      } else {
        // every product with this Q tile is complete: its shared memory is free
        good = mbar_wait_bounded(b_o + 8 * grp, 0);
        float* s_l = reinterpret_cast<float*>(base_ptr + grp * C::Q_BYTES);
        s_l[half * BQ + r] = l;
        mbar_arrive(xbar);
        good = mbar_wait_bounded(xbar, xphase) && good;
        l_other = s_l[(half ^ 1) * BQ + r];
      }
      if (!good) arcb_set_error(a.err, ARCB_DEV_WAIT_TIMEOUT_ACC);
      ok = __all_sync(0xffffffffu, good);
    }
    float l_row = half ? l_other + l : l + l_other;   // same order of addition in both threads
    float num = 1.f;
    if (a.sink && m_ref > -INFINITY) {
      const float d = __ldg(a.sink + h) * LOG2E - m_ref;
      if (d > 0.f) {      // bring both terms to the larger reference
        num = exp2f(-d);
        l_row = l_row * num + 1.f;
      } else {
        l_row += exp2f(d);
      }
    }
    const int qr = grp * BQ + r;
    const float inv = (ok && l_row > 0.f) ? num / l_row : 0.f;
    const size_t row = (size_t)row0 + qr;
    uint16_t* dst = reinterpret_cast<uint16_t*>(a.out) + (row * a.n_heads + h) * VP + half * (VP / 2);
    const uint16_t* gt = a.gate ? reinterpret_cast<const uint16_t*>(a.gate) + row * a.gate_pitch + (size_t)h * VP + half * (VP / 2) : nullptr;
#pragma unroll
    for (int c = 0; c < VP / 64; ++c) {
      uint32_t oreg[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) oreg[i] = 0u;
      if (ok && n_mine > j0) {
        tc_fence_after();
        tmem_ld_32x32(t_o + c * 32, oreg);
        tmem_wait_ld_dep(oreg);
      }
      if (qr < rows) {
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          float f[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(oreg[i + e]) * inv;
          if (gt) {
            const uint4 g4 = __ldg(reinterpret_cast<const uint4*>(gt + c * 32 + i));
            const uint32_t gw[4] = {g4.x, g4.y, g4.z, g4.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 g2 = unpack2_act(gw[e], F16 ? 1 : 0);
              f[2 * e] *= g2.x;
              f[2 * e + 1] *= g2.y;
            }
          }
          *reinterpret_cast<uint4*>(dst + c * 32 + i) =
              make_uint4(pack2_act(f[0], f[1], F16 ? 1 : 0), pack2_act(f[2], f[3], F16 ? 1 : 0),
                         pack2_act(f[4], f[5], F16 ? 1 : 0), pack2_act(f[6], f[7], F16 ? 1 : 0));
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, C::TMEM_COLS);
  }
}

template <int DP, int DR, int VP>
cudaError_t set_attr() {
  cudaError_t e = cudaFuncSetAttribute(attn_prefill_gqa_kernel<DP, DR, VP, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, FgCfg<DP, DR, VP>::SMEM);
  if (e != cudaSuccess) return e;
  return cudaFuncSetAttribute(attn_prefill_gqa_kernel<DP, DR, VP, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, FgCfg<DP, DR, VP>::SMEM);
}

template <int DP, int DR, int VP>
int launch(const AttnPrefillGqaArgs& a, cudaStream_t stream) {
  using C = FgCfg<DP, DR, VP>;
  CUtensorMap tq, tk, tv;
  const uint64_t cache_rows = (uint64_t)a.n_seqs * a.n_kv * a.t_max;
  const uint64_t kv_rows = DR > 0 ? (uint64_t)a.kv_rows : cache_rows;
  int r = arcb_make_tmap_2d_16b(&tq, a.q, (uint64_t)a.n_rows, (uint64_t)a.q_pitch, BQ, 64, a.act_f16);
  if (r) return 1000 + r;
  r = arcb_make_tmap_2d_16b(&tk, a.k, kv_rows, DR > 0 ? (uint64_t)a.kv_pitch : DP, BKV, 64, a.act_f16);
  if (r) return 1000 + r;
  r = arcb_make_tmap_2d_16b(&tv, a.v, kv_rows, DR > 0 ? (uint64_t)a.kv_pitch : VP, BKV, 64, a.act_f16);
  if (r) return 1000 + r;
  CUtensorMap tr = tk;
  if (DR > 0) {
    r = arcb_make_tmap_2d_16b(&tr, a.k_rot, (uint64_t)a.n_seqs * a.rot_panels * a.t_max, 64, BKV, 64, a.act_f16);
    if (r) return 1000 + r;
  }
  const int fmt = a.act_f16 ? 0 : 1;
  const uint32_t idesc_qk = umma_idesc_f16(BQ, BKV, fmt, fmt, 0, 0);
  const uint32_t idesc_pv = umma_idesc_f16(BQ, 64, fmt, fmt, 0, 1);   // V is MN-major, 64 columns a product
  const dim3 grid(a.n_heads, a.n_qblocks);
  const cudaError_t e =
      a.act_f16 ? arcb_launch(attn_prefill_gqa_kernel<DP, DR, VP, true>, grid, dim3(THREADS), C::SMEM, stream, tq, tk, tv, tr, a, idesc_qk, idesc_pv)
                : arcb_launch(attn_prefill_gqa_kernel<DP, DR, VP, false>, grid, dim3(THREADS), C::SMEM, stream, tq, tk, tv, tr, a, idesc_qk, idesc_pv);
  arcb_count_launch(1);
  return (int)e;
}

}  // namespace

bool arcb_attn_prefill_gqa_supported(int dimp, int vdimp, int n_seqs, int n_kv, int t_max, float scale) {
  // the reference maximum follows the largest raw score, which needs a positive scale
  return scale > 0.f && dimp <= 128 && vdimp <= 128 && (long long)n_seqs * n_kv * t_max < (1ll << 31) - 256;
}

bool arcb_attn_prefill_latent_supported(int dimp, int rotp, int vdimp, int panels, int n_seqs, int t_max, float scale) {
  return scale > 0.f && dimp <= 128 && rotp == 64 && vdimp <= 128 && (long long)n_seqs * panels * t_max < (1ll << 31) - 256;
}

int arcb_attn_prefill_gqa_init() {
  cudaError_t e;
  if ((e = set_attr<64, 0, 64>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<64, 0, 128>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<128, 0, 64>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<128, 0, 128>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<64, 64, 64>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<64, 64, 128>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<128, 64, 64>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<128, 64, 128>()) != cudaSuccess) return (int)e;
  return 0;
}

int arcb_launch_attn_prefill_gqa(const AttnPrefillGqaArgs& a, cudaStream_t stream) {
  if (a.n_qblocks <= 0) return 0;
  if (a.n_rows <= 0 || a.n_kv <= 0 || a.n_heads % a.n_kv || a.n_qblocks > 65535) return -1;
  if (a.kv0) {
    if (a.rotp != 64) return -1;
    switch (a.dimp * 1000 + a.vdimp) {
      case 64064: return launch<64, 64, 64>(a, stream);
      case 64128: return launch<64, 64, 128>(a, stream);
      case 128064: return launch<128, 64, 64>(a, stream);
      case 128128: return launch<128, 64, 128>(a, stream);
    }
    return -1;
  }
  switch (a.dimp * 1000 + a.vdimp) {
    case 64064: return launch<64, 0, 64>(a, stream);
    case 64128: return launch<64, 0, 128>(a, stream);
    case 128064: return launch<128, 0, 64>(a, stream);
    case 128128: return launch<128, 0, 128>(a, stream);
  }
  return -1;
}
