// Decode attention over cached latents on tcgen05 tensor cores, keys as the rows of every product.
//
// All heads of a sequence read the same cached rows, so a row is loaded once and multiplied with up to NH queries.
// A work unit is one item (query row) x one block of NH heads x one split of its visible rows; persistent CTAs take
// units one after the other, loads running ahead across unit borders.  Per tile of KEYS cached rows:
//   TMA      latent columns as boxes of KEYS rows x 64 columns, two boxes (128 columns) to a ring slot; the rotated
//            part in a box of its own
//   MMA      S^T [KEYS x NH heads] = rows . Q^T (both operands K-major), fp32 in NH TMEM columns
//   softmax  a thread owns one key: NH scores.  Reference maxima per head live in shared memory and are raised only
//            when a tile exceeds one by 2^8 (then the sums and O are rescaled), so the usual tile needs no exchange of
//            maxima; p = exp2(s c - m) in fp32, sums per thread in fp32, P in the operand format as a row of NH
//            columns (an MN-major operand)
//   MMA      O^T [128 latent columns x NH heads] += C^T P for every ring slot, C^T being the very bytes that were the
//            row operand before (MN-major), then the slot goes back to the producer
// The latents therefore cross HBM and shared memory once for both products.  Two groups of softmax warps take the
// tiles of a unit in turn, each with scores, P, sums, maxima and O of its own, so that a tile's scores are multiplied
// while the other tile is in its softmax; the groups' results are merged at the unit's end, where the denominators are
// summed over threads and a sink joins them.  Splits leave unnormalised sums for arcb_launch_attn_combine.  KEYS is 128
// where the ring then holds two tiles, else 64.  Every wait is bounded.
#include "attn_gqa.cuh"
#include "attn_latent.cuh"
#include "flash_common.cuh"
#include "gemm.cuh"
#include "launch.cuh"

using namespace sm100;

namespace {

constexpr int THREADS = 352;                 // producer, one issuer per product, two groups of four softmax warps
constexpr int MAX_SLOTS = 16;
constexpr int TMEM_COLS = 512;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float RAISE = 8.f;                 // log2 units
constexpr int STATIC_SMEM = 4096;            // bound of the kernel's static shared memory

struct Carve {                               // byte offsets from the aligned start
  int q, rot, p, ring, bars, total;
};
__host__ __device__ inline Carve carve(int kvp, int nh, int keys, int slots) {
  const int box = keys * 128;
  Carve c;
  c.q = 0;
  c.rot = (kvp / 64 + 1) * nh * 128;
  c.p = c.rot + 2 * box;
  c.ring = c.p + box;                        // both groups' P share the 128-byte rows
  c.bars = c.ring + slots * 2 * box;
  c.total = c.bars + 512;
  return c;
}
int ring_slots(int kvp, int nh, int keys) {
  const int n = (227 * 1024 - STATIC_SMEM - 1024 - carve(kvp, nh, keys, 0).total) / (keys * 256);
  return n > MAX_SLOTS ? MAX_SLOTS : n;
}
int heads_of_block(int n_heads) { return n_heads <= 16 ? 16 : 32; }
int keys_of_tile(int kvp, int nh) { return ring_slots(kvp, nh, 128) >= 2 * (kvp / 128) ? 128 : 64; }

// MN-major operand of two 64-element groups `box` bytes apart (rows of 128 bytes, 128-byte swizzle)
__device__ __forceinline__ uint64_t desc_mn_pair(uint32_t addr, uint32_t box) {
  uint64_t d = 0;
  d |= (uint64_t)((addr & 0x3FFFFu) >> 4);
  d |= (uint64_t)(box >> 4) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

template <int NH>
__device__ __forceinline__ void ld_heads(uint32_t addr, uint32_t (&r)[NH]) {
  if constexpr (NH == 16) tmem_ld_32x16(addr, r);
  else {
#pragma unroll
    for (int g = 0; g < NH / 32; ++g) tmem_ld_32x32(addr + g * 32, *reinterpret_cast<uint32_t (*)[32]>(&r[g * 32]));
  }
  tmem_wait_ld();
}
template <int NH>
__device__ __forceinline__ void st_heads(uint32_t addr, const uint32_t (&r)[NH]) {
  if constexpr (NH == 16) tmem_st_32x16(addr, r);
  else {
#pragma unroll
    for (int g = 0; g < NH / 32; ++g) tmem_st_32x32(addr + g * 32, *reinterpret_cast<const uint32_t (*)[32]>(&r[g * 32]));
  }
}

// Reduces N values per lane over the warp's lanes: lane i returns the result of value i / (32 / N).
template <int N, typename Op>
__device__ __forceinline__ float reduce_columns(float* v, int lane, Op op) {
#pragma unroll
  for (int st = N / 2; st >= 1; st >>= 1) {
    const int dist = st * (32 / N);
    const bool up = (lane & dist) != 0;
#pragma unroll
    for (int j = 0; j < st; ++j) {
      const float send = up ? v[j] : v[j + st];
      const float keep = up ? v[j + st] : v[j];
      v[j] = op(keep, __shfl_xor_sync(0xffffffffu, send, dist));
    }
  }
#pragma unroll
  for (int dist = 32 / N / 2; dist >= 1; dist >>= 1) v[0] = op(v[0], __shfl_xor_sync(0xffffffffu, v[0], dist));
  return v[0];
}

struct Unit {
  int item, hb, split, seq, begin, tiles, end;   // tiles < 0: no unit
};
template <int KEYS>
__device__ __forceinline__ Unit unit_of(const AttnLatentArgs& a, int w, int head_blocks, int total) {
  Unit u;
  if (w >= total) {
    u.tiles = -1;
    return u;
  }
  u.hb = w % head_blocks; w /= head_blocks;      // blocks of one item side by side: they share its rows in L2
  u.split = w % a.n_splits;
  u.item = w / a.n_splits;
  u.seq = a.item_seq ? a.item_seq[u.item] : u.item;
  int len = a.item_len[u.item];
  if (len > a.t_max || u.seq < 0 || u.seq >= a.n_seqs) {
    arcb_set_error(a.err, ARCB_DEV_BAD_INDEX);
    len = 0;
  }
  len = max(len, 0);
  u.begin = a.window > 0 ? max(0, len - a.window) : 0;
  u.end = len;
  if (a.n_splits > 1) {
    const int chunk = ((u.end - u.begin + a.n_splits - 1) / a.n_splits + KEYS - 1) / KEYS * KEYS;
    u.begin = min(u.begin + u.split * chunk, len);
    u.end = min(u.begin + chunk, len);
  }
  u.tiles = (u.end - u.begin + KEYS - 1) / KEYS;
  return u;
}

template <int NH, int KEYS, bool F16>
__global__ void __launch_bounds__(THREADS, 1)
attn_latent_tc_kernel(const __grid_constant__ CUtensorMap tmap_c, const __grid_constant__ CUtensorMap tmap_ql,
                      const __grid_constant__ CUtensorMap tmap_qr, AttnLatentArgs a, uint32_t idesc_s, uint32_t idesc_o,
                      int slots, int head_blocks, int total) {
  constexpr int BOX = KEYS * 128, SLOT = 2 * BOX;
  constexpr int LANES = KEYS / 4;                // lanes of a softmax warp that own a key
  pdl_launch_dependents();
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  __shared__ float s_wmax[2][4][NH], s_l[2][4][NH], s_ref[2][NH], s_alpha[2][NH], s_f[2][NH];
  __shared__ uint32_t s_tmem;
  static_assert(sizeof(float) * 22 * NH + 64 <= STATIC_SMEM, "static shared memory");
  const uint32_t raw = smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - raw);
  const Carve cv = carve(a.kvp, NH, KEYS, slots);
  // one barrier each: queries full / empty; two each: rotated box full / empty, scores, P written, P read (per
  // group); one each: O complete, O read; then the ring
  const uint32_t b_qf = base + cv.bars, b_qe = b_qf + 8, b_rf = b_qf + 16, b_re = b_rf + 16, b_s = b_re + 16, b_p = b_s + 16,
                 b_pv = b_p + 16, b_o = b_pv + 16, b_or = b_o + 8, b_uf = b_or + 8, b_ue = b_uf + 8 * MAX_SLOTS;
  const int warp = __shfl_sync(0xffffffffu, (int)threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  const int n_d = a.kvp / 128;

  if (threadIdx.x == 0) {
    mbar_init(b_qf, 1);
    mbar_init(b_qe, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(b_rf + 8 * i, 1);
      mbar_init(b_re + 8 * i, 1);
      mbar_init(b_s + 8 * i, 1);
      mbar_init(b_p + 8 * i, 128);
      mbar_init(b_pv + 8 * i, 1);
    }
    mbar_init(b_o, 1);
    mbar_init(b_or, 256);
    for (int i = 0; i < slots; ++i) {
      mbar_init(b_uf + 8 * i, 1);
      mbar_init(b_ue + 8 * i, 1);
    }
    mbar_fence_init();
    tma_prefetch_desc(&tmap_c);
    tma_prefetch_desc(&tmap_ql);
    tma_prefetch_desc(&tmap_qr);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&s_tmem), TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t t_s = __shfl_sync(0xffffffffu, s_tmem, 0), t_o = t_s + 2 * NH;   // scores of group g at t_s + g NH, O at t_o + g n_d NH
  pdl_wait();

  if (warp == 0) {
    if (lane == 0) {
      // ---- TMA producer ----
      int n = 0, t = 0, q = 0;     // ring slots, tiles and units so far
      bool ok = true;
      auto wait = [&](uint32_t bar, uint32_t parity) {
        if (ok && !mbar_wait_bounded(bar, parity)) {
          arcb_set_error(a.err, ARCB_DEV_WAIT_TIMEOUT_MMA);
          ok = false;
        }
        return ok;
      };
      int w = blockIdx.x;
      Unit next = unit_of<KEYS>(a, w, head_blocks, total);
      while (ok && next.tiles >= 0) {
        const Unit u = next;
        w += gridDim.x;
        next = unit_of<KEYS>(a, w, head_blocks, total);       // its loads are in flight while this unit is worked on
        if (!u.tiles) continue;
        const int row0 = u.seq * (2 * n_d + 1) * a.t_max + u.begin;     // of the first panel
        for (int j = 0; ok && j < u.tiles; ++j, ++t) {
          for (int d = 0; d < n_d; ++d, ++n) {
            const int s = n % slots;
            if (!wait(b_ue + 8 * s, ((n / slots) & 1) ^ 1)) break;
            mbar_expect_tx(b_uf + 8 * s, SLOT);
            const uint32_t dst = base + cv.ring + s * SLOT;
            tma_load_2d(dst, &tmap_c, 0, row0 + 2 * d * a.t_max + j * KEYS, b_uf + 8 * s);
            tma_load_2d(dst + BOX, &tmap_c, 0, row0 + (2 * d + 1) * a.t_max + j * KEYS, b_uf + 8 * s);
          }
          const int rb = t & 1;
          if (!wait(b_re + 8 * rb, ((t >> 1) & 1) ^ 1)) break;
          mbar_expect_tx(b_rf + 8 * rb, BOX);
          tma_load_2d(base + cv.rot + rb * BOX, &tmap_c, 0, row0 + 2 * n_d * a.t_max + j * KEYS, b_rf + 8 * rb);
          if (j == 0) {            // behind the first tile: its rows do not wait for the last unit's scores
            if (!wait(b_qe, (q & 1) ^ 1)) break;
            const int qrow = u.item * a.n_heads + u.hb * NH;
            mbar_expect_tx(b_qf, (2 * n_d + 1) * NH * 128);
            for (int c = 0; c < 2 * n_d; ++c) tma_load_2d(base + cv.q + c * NH * 128, &tmap_ql, c * 64, qrow, b_qf);
            tma_load_2d(base + cv.q + 2 * n_d * NH * 128, &tmap_qr, a.q_off, qrow, b_qf);
          }
        }
        ++q;
      }
    }
  } else if (warp < 3) {
    // ---- MMA issuers, the whole warp with one elected lane: warp 1 scores, warp 2 the products with P ----
    const uint32_t el = elect_one();
    int n = 0, t = 0, q = 0;
    int uses[2] = {0, 0};          // tiles of each group so far
    bool ok = true;
    auto wait = [&](uint32_t bar, uint32_t parity, int code) {
      if (ok && !__all_sync(0xffffffffu, mbar_wait_bounded(bar, parity))) {
        arcb_set_error(a.err, code);
        ok = false;
      }
      return ok;
    };
    int w = blockIdx.x;
    Unit next = unit_of<KEYS>(a, w, head_blocks, total);
    while (ok && next.tiles >= 0) {
      const Unit u = next;
      w += gridDim.x;
      next = unit_of<KEYS>(a, w, head_blocks, total);
      if (!u.tiles) continue;
      if (warp == 1 && !wait(b_qf, q & 1, ARCB_DEV_WAIT_TIMEOUT_TMA)) break;
      for (int j = 0; ok && j < u.tiles; ++j, ++t) {
        const int g = j & 1;
        if (warp == 1) {
          // the group has read the scores this tile overwrites
          if (!wait(b_p + 8 * g, (uses[g] & 1) ^ 1, ARCB_DEV_WAIT_TIMEOUT_ACC)) break;
          for (int d = 0; d < n_d; ++d, ++n) {
            const int s = n % slots;
            if (!wait(b_uf + 8 * s, (n / slots) & 1, ARCB_DEV_WAIT_TIMEOUT_TMA)) break;
            tc_fence_after();
#pragma unroll
            for (int b = 0; b < 2; ++b) {
              const uint64_t dk = umma_desc_k_sw128(base + cv.ring + s * SLOT + b * BOX);
              const uint64_t dq = umma_desc_k_sw128(base + cv.q + (2 * d + b) * NH * 128);
#pragma unroll
              for (int ks = 0; ks < 4; ++ks) umma_f16_if(el, t_s + g * NH, dk + 2 * ks, dq + 2 * ks, idesc_s, (d | b | ks) ? 1u : 0u);
            }
          }
          const int rb = t & 1;
          if (!wait(b_rf + 8 * rb, (t >> 1) & 1, ARCB_DEV_WAIT_TIMEOUT_TMA)) break;
          tc_fence_after();
          const uint64_t dk = umma_desc_k_sw128(base + cv.rot + rb * BOX);
          const uint64_t dq = umma_desc_k_sw128(base + cv.q + 2 * n_d * NH * 128);
#pragma unroll
          for (int ks = 0; ks < 4; ++ks) umma_f16_if(el, t_s + g * NH, dk + 2 * ks, dq + 2 * ks, idesc_s, 1u);
          umma_commit_if(el, b_re + 8 * rb);
          if (j + 1 == u.tiles) umma_commit_if(el, b_qe);
          umma_commit_if(el, b_s + 8 * g);
        } else {
          if (!wait(b_p + 8 * g, uses[g] & 1, ARCB_DEV_WAIT_TIMEOUT_ACC)) break;
          // both groups have read O of the unit before
          if (j < 2 && !wait(b_or, (q & 1) ^ 1, ARCB_DEV_WAIT_TIMEOUT_ACC)) break;
          const uint64_t dp = umma_desc_mn_sw128(base + cv.p + g * 64);
          for (int d = 0; d < n_d; ++d, ++n) {
            const int s = n % slots;
            if (!wait(b_uf + 8 * s, (n / slots) & 1, ARCB_DEV_WAIT_TIMEOUT_TMA)) break;   // long since there
            tc_fence_after();
            const uint64_t dc = desc_mn_pair(base + cv.ring + s * SLOT, BOX);
#pragma unroll
            for (int ks = 0; ks < KEYS / 16; ++ks)
              umma_f16_if(el, t_o + (g * n_d + d) * NH, dc + ks * (2048 >> 4), dp + ks * (2048 >> 4), idesc_o, (j > 1 || ks) ? 1u : 0u);
            umma_commit_if(el, b_ue + 8 * s);
          }
          umma_commit_if(el, b_pv + 8 * g);
          if (j + 1 == u.tiles) umma_commit_if(el, b_o);
        }
        ++uses[g];
      }
      ++q;
    }
  } else {
    // ---- softmax and output: key (then latent column) of lane and quarter ----
    const int quarter = warp & 3, g = (warp - 3) >> 2;
    const int key = quarter * LANES + lane, col = quarter * 32 + lane;
    const bool owner = lane < LANES;
    const uint32_t lane_off = (uint32_t)(quarter * 32) << 16;
    const int h_mine = (int)threadIdx.x - 96 - g * 128;      // the head whose bookkeeping this thread does, if < NH
    const int bar_id = 1 + g;
    const float sc = a.scale * LOG2E;
    const uint32_t t_sg = t_s + g * NH + lane_off, t_og = t_o + g * n_d * NH + lane_off;
    uint8_t* my_p = base_ptr + cv.p + key * 128;
    int uses = 0, q = 0;
    int w = blockIdx.x;
    Unit next = unit_of<KEYS>(a, w, head_blocks, total);
    while (next.tiles >= 0) {
      const Unit u = next;
      w += gridDim.x;
      next = unit_of<KEYS>(a, w, head_blocks, total);
      const int h0 = u.hb * NH, nh = min(NH, a.n_heads - h0);
      const size_t ih0 = (size_t)u.item * a.n_heads + h0;
      const float my_sink = a.n_splits == 1 && a.sink && h_mine < nh ? __ldg(a.sink + h0 + h_mine) * LOG2E : -INFINITY;
      float l[NH];
#pragma unroll
      for (int h = 0; h < NH; ++h) l[h] = 0.f;
      bool ok = true;
      for (int j = g; j < u.tiles; j += 2, ++uses) {
        // its scores are there, and its last product with P is complete: P and O may be written
        ok = mbar_wait_bounded(b_s + 8 * g, uses & 1) && mbar_wait_bounded(b_pv + 8 * g, (uses & 1) ^ 1);
        ok = !named_bar_or(bar_id, 128, !ok);
        if (!ok) break;
        tc_fence_after();
        const bool first = j < 2;
        const bool seen = owner && u.begin + j * KEYS + key < u.end;
        float wm;
        {
          uint32_t sv[NH];
          ld_heads<NH>(t_sg, sv);
          float v[NH];
#pragma unroll
          for (int h = 0; h < NH; ++h) v[h] = seen ? __uint_as_float(sv[h]) * sc : -INFINITY;
          wm = reduce_columns<NH>(v, lane, [](float x, float y) { return fmaxf(x, y); });
        }
        const int my_h = lane / (32 / NH);
        const bool raise = first || wm > s_ref[g][my_h] + RAISE;
        s_wmax[g][quarter][my_h] = wm;
        if (named_bar_or(bar_id, 128, raise)) {
          if (h_mine < NH) {
            const float* m4 = &s_wmax[g][0][h_mine];
            float mx = fmaxf(fmaxf(m4[0], m4[NH]), fmaxf(m4[2 * NH], m4[3 * NH]));
            const float old = first ? -INFINITY : s_ref[g][h_mine];
            if (!(mx > old + RAISE)) mx = old;
            s_alpha[g][h_mine] = first ? 0.f : exp2f(old - mx);
            s_ref[g][h_mine] = mx;
          }
          named_bar_sync(bar_id, 128);
          if (!first) {
#pragma unroll
            for (int h = 0; h < NH; ++h) l[h] *= s_alpha[g][h];
            for (int d = 0; d < n_d; ++d) {
              uint32_t o[NH];
              ld_heads<NH>(t_og + d * NH, o);
#pragma unroll
              for (int h = 0; h < NH; ++h) o[h] = __float_as_uint(__uint_as_float(o[h]) * s_alpha[g][h]);
              st_heads<NH>(t_og + d * NH, o);
            }
            tmem_wait_st();
          }
        }
        {
          uint32_t sv[NH];
          ld_heads<NH>(t_sg, sv);
#pragma unroll
          for (int c = 0; c < NH / 8; ++c) {
            if (c * 8 >= nh) break;            // columns of heads that do not exist stay what they are
            uint32_t pk[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int h = c * 8 + 2 * e;
              const float2 ref = *reinterpret_cast<const float2*>(&s_ref[g][h]);
              const float p0 = seen ? ex2_fast(fmaf(__uint_as_float(sv[h]), sc, -ref.x)) : 0.f;
              const float p1 = seen ? ex2_fast(fmaf(__uint_as_float(sv[h + 1]), sc, -ref.y)) : 0.f;
              l[h] += p0;
              l[h + 1] += p1;
              pk[e] = pack2_prob(p0, p1, F16 ? 1 : 0);
            }
            if (owner) *reinterpret_cast<uint4*>(my_p + (((c + 4 * g) ^ (key & 7)) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
          }
        }
        fence_proxy_async_smem();
        tc_fence_before();
        mbar_arrive(b_p + 8 * g);
      }
      if (ok && u.tiles) {
        ok = mbar_wait_bounded(b_o, q & 1);
        ++q;
      }
      ok = !named_bar_or(3, 256, !ok);
      if (!ok) {
        arcb_set_error(a.err, ARCB_DEV_WAIT_TIMEOUT_ACC);
        break;
      }
      // denominators: over the lanes, then over the warps in a fixed order, then the two groups
      s_l[g][quarter][lane / (32 / NH)] = reduce_columns<NH>(l, lane, [](float x, float y) { return x + y; });
      named_bar_sync(3, 256);
      if (g == 0 && h_mine < NH) {
        const int h = h_mine;
        float lg[2], ref[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          lg[i] = (s_l[i][0][h] + s_l[i][1][h]) + (s_l[i][2][h] + s_l[i][3][h]);
          ref[i] = u.tiles > i ? s_ref[i][h] : -INFINITY;
        }
        const bool last = a.n_splits == 1;
        const float sk = u.tiles ? my_sink : -INFINITY;
        const float m = fmaxf(fmaxf(ref[0], ref[1]), sk);
        const float ms = m == -INFINITY ? 0.f : m;
        float f[2] = {exp2f(ref[0] - ms), exp2f(ref[1] - ms)};
        const float lt = lg[0] * f[0] + lg[1] * f[1] + exp2f(sk - ms);
        if (!last && h < nh) {
          float* rec = a.scratch + ((ih0 + h) * a.n_splits + u.split) * (a.kvp + 4);
          rec[a.kvp] = m;
          rec[a.kvp + 1] = lt;
        }
        const float inv = last ? (lt > 0.f ? 1.f / lt : 0.f) : 1.f;
        s_f[0][h] = f[0] * inv;
        s_f[1][h] = f[1] * inv;
      }
      named_bar_sync(3, 256);
      tc_fence_after();
      for (int d = g; d < n_d; d += 2) {     // both groups' sums of every second block of columns
        float o[NH];
#pragma unroll
        for (int h = 0; h < NH; ++h) o[h] = 0.f;
        for (int i = 0; i < min(u.tiles, 2); ++i) {
          uint32_t part[NH];
          ld_heads<NH>(t_o + (i * n_d + d) * NH + lane_off, part);
#pragma unroll
          for (int h = 0; h < NH; ++h) o[h] = fmaf(__uint_as_float(part[h]), s_f[i][h], o[h]);
        }
#pragma unroll
        for (int h = 0; h < NH; ++h) {
          if (h >= nh) break;
          if (a.n_splits > 1) a.scratch[((ih0 + h) * a.n_splits + u.split) * (a.kvp + 4) + d * 128 + col] = o[h];
          else st_act(a.out, (ih0 + h) * a.kvp + d * 128 + col, o[h], F16 ? 1 : 0);
        }
      }
      tc_fence_before();
      if (u.tiles) mbar_arrive(b_or);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(s_tmem, TMEM_COLS);
  }
}

template <int NH, int KEYS>
cudaError_t set_attr() {
  const int bytes = 227 * 1024 - STATIC_SMEM;
  cudaError_t e = cudaFuncSetAttribute(attn_latent_tc_kernel<NH, KEYS, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return e;
  return cudaFuncSetAttribute(attn_latent_tc_kernel<NH, KEYS, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
}

template <int NH, int KEYS>
int launch(const AttnLatentArgs& a, cudaStream_t stream) {
  CUtensorMap tc, tl, tr;
  const int f16 = a.fmt == 1;
  const uint64_t qrows = (uint64_t)a.n_items * a.n_heads;
  int r = arcb_make_tmap_2d_16b(&tc, a.cache, (uint64_t)a.n_seqs * ((a.kvp + a.rotp) / 64) * a.t_max, 64, KEYS, 64, f16);
  if (!r) r = arcb_make_tmap_2d_16b(&tl, a.qlat, qrows, (uint64_t)a.kvp, NH, 64, f16);
  if (!r) r = arcb_make_tmap_2d_16b(&tr, a.q, qrows, (uint64_t)a.q_head, NH, 64, f16);
  if (r) return 1000 + r;
  const int slots = ring_slots(a.kvp, NH, KEYS), hb = (a.n_heads + NH - 1) / NH;
  if (slots < a.kvp / 128) return -1;             // a tile must fit
  const long long total = (long long)a.n_items * a.n_splits * hb;
  if (total > 0x7fffffffLL) return -1;
  const int fmt = f16 ? 0 : 1;
  const uint32_t is = umma_idesc_f16(KEYS, NH, fmt, fmt, 0, 0), io = umma_idesc_f16(128, NH, fmt, fmt, 1, 1);
  const dim3 grid((unsigned)(total < 148 ? total : 148));
  const size_t smem = carve(a.kvp, NH, KEYS, slots).total + 1024;
  const cudaError_t e = f16 ? arcb_launch(attn_latent_tc_kernel<NH, KEYS, true>, grid, dim3(THREADS), smem, stream, tc, tl, tr, a, is, io, slots, hb, (int)total)
                            : arcb_launch(attn_latent_tc_kernel<NH, KEYS, false>, grid, dim3(THREADS), smem, stream, tc, tl, tr, a, is, io, slots, hb, (int)total);
  arcb_count_launch(1);
  return (int)e;
}

}  // namespace

bool arcb_attn_latent_tc_supported(int kvp, int rotp, int fmt, int n_seqs, int t_max, float scale) {
  // the reference maxima follow the largest raw score, which needs a positive scale
  return fmt != 2 && scale > 0.f && kvp % 128 == 0 && kvp <= 512 && rotp == 64 &&
         (long long)n_seqs * (kvp / 64 + 1) * t_max < (1ll << 31) - 256;
}

int arcb_attn_latent_splits(int n_items, int n_heads, int kvp, int keys) {
  // one unit per SM at least, none shorter than 256 keys
  const int nh = heads_of_block(n_heads);
  const long long units = (long long)n_items * ((n_heads + nh - 1) / nh);
  long long s = 148 / (units < 1 ? 1 : units);
  const long long most = (keys + 255) / 256;
  if (keys > 0 && s > most) s = most;
  if (s > 32) s = 32;
  return s < 1 ? 1 : (int)s;
}

int arcb_attn_latent_init() {
  cudaError_t e;
  if ((e = set_attr<16, 64>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<16, 128>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<32, 64>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<32, 128>()) != cudaSuccess) return (int)e;
  return 0;
}

int arcb_launch_attn_latent_tc(const AttnLatentArgs& a, cudaStream_t stream) {
  if (a.n_items <= 0) return 0;
  if (!arcb_attn_latent_tc_supported(a.kvp, a.rotp, a.fmt, a.n_seqs, a.t_max, a.scale) || a.q_off % 8 || a.q_head % 8) return -1;
  if (a.n_splits < 1 || (a.n_splits > 1 && !a.scratch)) return -1;
  const int nh = heads_of_block(a.n_heads), keys = keys_of_tile(a.kvp, nh);
  const int r = nh == 16 ? (keys == 64 ? launch<16, 64>(a, stream) : launch<16, 128>(a, stream))
                         : (keys == 64 ? launch<32, 64>(a, stream) : launch<32, 128>(a, stream));
  if (r || a.n_splits == 1) return r;
  AttnGqaArgs c{};
  c.out = a.out; c.sink = a.sink; c.n_items = a.n_items; c.n_heads = a.n_heads; c.vdimp = a.kvp; c.n_splits = a.n_splits;
  c.scratch = a.scratch; c.fmt = a.fmt;
  return arcb_launch_attn_combine(c, stream);
}
