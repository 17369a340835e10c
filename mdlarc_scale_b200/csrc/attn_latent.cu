// Decode attention over cached latents on tcgen05 tensor cores, keys as the rows of every product.
//
// All heads of a sequence read the same cached rows, so a row is loaded once and multiplied with up to NH queries.
// A work unit is one item (query row) x one block of NH heads x one split of its visible rows; persistent CTAs take
// units one after the other, loads running ahead across unit borders.  Per tile of 128 cached rows:
//   TMA      latent columns as boxes of 128 rows x 64 columns, two boxes (128 columns) to a ring slot; the rotated
//            part in a box of its own
//   MMA      S^T [128 keys x NH heads] = rows . Q^T (both operands K-major), fp32 in NH TMEM columns
//   softmax  a thread owns one key: NH scores.  Reference maxima per head live in shared memory and are raised only
//            when a tile exceeds one by 2^8 (then the sums and O are rescaled), so the usual tile needs no exchange of
//            maxima; p = exp2(s c - m) in fp32, sums per thread in fp32, P in the operand format as a row of NH
//            columns (an MN-major operand)
//   MMA      O^T [128 latent columns x NH heads] += C^T P for every ring slot, C^T being the very bytes that were the
//            row operand before (MN-major), then the slot goes back to the producer
// The latents therefore cross HBM and shared memory once for both products.  Denominators are summed over threads at
// the end; a sink only joins them.  Splits leave unnormalised sums for arcb_launch_attn_combine.  Every wait is bounded.
#include "attn_gqa.cuh"
#include "attn_latent.cuh"
#include "flash_common.cuh"
#include "gemm.cuh"
#include "launch.cuh"

using namespace sm100;

namespace {

constexpr int THREADS = 192;                 // producer, MMA issuer, four softmax warps
constexpr int KEYS = 128;
constexpr int BOX = KEYS * 128;              // 128 rows x 64 16-bit columns
constexpr int SLOT = 2 * BOX;
constexpr int MAX_SLOTS = 8;
constexpr int TMEM_COLS = 256;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float RAISE = 8.f;                 // log2 units
constexpr int STATIC_SMEM = 4096;            // bound of the kernel's static shared memory

struct Carve {                               // byte offsets from the aligned start
  int q, rot, p, ring, bars, total;
};
__host__ __device__ inline Carve carve(int kvp, int nh, int slots) {
  Carve c;
  c.q = 0;
  c.rot = (kvp / 64 + 1) * nh * 128;
  c.p = c.rot + BOX;
  c.ring = c.p + BOX;
  c.bars = c.ring + slots * SLOT;
  c.total = c.bars + 256;
  return c;
}
int ring_slots(int kvp, int nh) {
  const int n = (227 * 1024 - STATIC_SMEM - 1024 - carve(kvp, nh, 0).total) / SLOT;
  return n > MAX_SLOTS ? MAX_SLOTS : n;
}
int heads_of_block(int n_heads, int kvp) {
  if (n_heads <= 16) return 16;
  return n_heads > 32 && kvp <= 256 ? 64 : 32;
}

// MN-major operand of two 64-element groups BOX bytes apart (rows of 128 bytes, 128-byte swizzle)
__device__ __forceinline__ uint64_t desc_mn_pair(uint32_t addr) {
  uint64_t d = 0;
  d |= (uint64_t)((addr & 0x3FFFFu) >> 4);
  d |= (uint64_t)(BOX >> 4) << 16;
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
  int item, hb, split, seq, begin, tiles, end;
};
__device__ __forceinline__ Unit unit_of(const AttnLatentArgs& a, int w, int head_blocks) {
  Unit u;
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

template <int NH, bool F16>
__global__ void __launch_bounds__(THREADS, 1)
attn_latent_tc_kernel(const __grid_constant__ CUtensorMap tmap_c, const __grid_constant__ CUtensorMap tmap_ql,
                      const __grid_constant__ CUtensorMap tmap_qr, AttnLatentArgs a, uint32_t idesc_s, uint32_t idesc_o,
                      int slots, int head_blocks, int total) {
  constexpr int G = NH / 32 > 0 ? NH / 32 : 1;   // values a lane holds after a reduction over lanes
  constexpr int N1 = NH < 32 ? NH : 32;
  pdl_launch_dependents();
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  __shared__ float s_wmax[4][NH], s_l[4][NH], s_ref[NH], s_alpha[NH], s_inv[NH];
  __shared__ uint32_t s_tmem;
  static_assert(sizeof(float) * 11 * NH + 64 <= STATIC_SMEM, "static shared memory");
  const uint32_t raw = smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - raw);
  const Carve cv = carve(a.kvp, NH, slots);
  const uint32_t b_qf = base + cv.bars, b_qe = b_qf + 8, b_rf = b_qf + 16, b_re = b_qf + 24, b_s = b_qf + 32, b_p = b_qf + 40,
                 b_o = b_qf + 48, b_uf = b_qf + 64, b_ue = b_uf + 8 * MAX_SLOTS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n_d = a.kvp / 128;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 7; ++i) mbar_init(b_qf + 8 * i, b_qf + 8 * i == b_p ? 128 : 1);
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
  const uint32_t t_s = s_tmem, t_o = t_s + NH;
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
      for (int w = blockIdx.x; ok && w < total; w += gridDim.x) {
        const Unit u = unit_of(a, w, head_blocks);
        if (!u.tiles) continue;
        if (!wait(b_qe, (q & 1) ^ 1)) break;
        const int qrow = u.item * a.n_heads + u.hb * NH;
        mbar_expect_tx(b_qf, (2 * n_d + 1) * NH * 128);
        for (int c = 0; c < 2 * n_d; ++c) tma_load_2d(base + cv.q + c * NH * 128, &tmap_ql, c * 64, qrow, b_qf);
        tma_load_2d(base + cv.q + 2 * n_d * NH * 128, &tmap_qr, a.q_off, qrow, b_qf);
        const int row0 = u.seq * a.t_max + u.begin;
        for (int j = 0; j < u.tiles; ++j, ++t) {
          for (int d = 0; d < n_d; ++d, ++n) {
            const int s = n % slots;
            if (!wait(b_ue + 8 * s, ((n / slots) & 1) ^ 1)) break;
            mbar_expect_tx(b_uf + 8 * s, SLOT);
            const uint32_t dst = base + cv.ring + s * SLOT;
            tma_load_2d(dst, &tmap_c, d * 128, row0 + j * KEYS, b_uf + 8 * s);
            tma_load_2d(dst + BOX, &tmap_c, d * 128 + 64, row0 + j * KEYS, b_uf + 8 * s);
          }
          if (!wait(b_re, (t & 1) ^ 1)) break;
          mbar_expect_tx(b_rf, BOX);
          tma_load_2d(base + cv.rot, &tmap_c, a.kvp, row0 + j * KEYS, b_rf);
        }
        ++q;
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      // ---- MMA issuer ----
      int n = 0, t = 0, q = 0;
      bool ok = true;
      auto wait = [&](uint32_t bar, uint32_t parity, int code) {
        if (ok && !mbar_wait_bounded(bar, parity)) {
          arcb_set_error(a.err, code);
          ok = false;
        }
        return ok;
      };
      for (int w = blockIdx.x; ok && w < total; w += gridDim.x) {
        const Unit u = unit_of(a, w, head_blocks);
        if (!u.tiles) continue;
        if (!wait(b_qf, q & 1, ARCB_DEV_WAIT_TIMEOUT_TMA)) break;
        for (int j = 0; ok && j < u.tiles; ++j, ++t) {
          for (int d = 0; d < n_d; ++d) {
            const int s = (n + d) % slots;
            if (!wait(b_uf + 8 * s, ((n + d) / slots) & 1, ARCB_DEV_WAIT_TIMEOUT_TMA)) break;
            tc_fence_after();
#pragma unroll
            for (int b = 0; b < 2; ++b) {
              const uint64_t dk = umma_desc_k_sw128(base + cv.ring + s * SLOT + b * BOX);
              const uint64_t dq = umma_desc_k_sw128(base + cv.q + (2 * d + b) * NH * 128);
#pragma unroll
              for (int ks = 0; ks < 4; ++ks) umma_f16(t_s, dk + 2 * ks, dq + 2 * ks, idesc_s, (d | b | ks) ? 1u : 0u);
            }
          }
          if (!wait(b_rf, t & 1, ARCB_DEV_WAIT_TIMEOUT_TMA)) break;
          tc_fence_after();
          {
            const uint64_t dk = umma_desc_k_sw128(base + cv.rot);
            const uint64_t dq = umma_desc_k_sw128(base + cv.q + 2 * n_d * NH * 128);
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) umma_f16(t_s, dk + 2 * ks, dq + 2 * ks, idesc_s, 1u);
          }
          umma_commit(b_re);
          if (j + 1 == u.tiles) umma_commit(b_qe);
          umma_commit(b_s);
          if (!wait(b_p, t & 1, ARCB_DEV_WAIT_TIMEOUT_ACC)) break;
          tc_fence_after();
          const uint64_t dp = umma_desc_mn_sw128(base + cv.p);
          for (int d = 0; d < n_d; ++d) {
            const int s = (n + d) % slots;
            const uint64_t dc = desc_mn_pair(base + cv.ring + s * SLOT);
#pragma unroll
            for (int ks = 0; ks < KEYS / 16; ++ks)
              umma_f16(t_o + d * NH, dc + ks * (2048 >> 4), dp + ks * (2048 >> 4), idesc_o, (j | ks) ? 1u : 0u);
            umma_commit(b_ue + 8 * s);
          }
          n += n_d;
        }
        if (ok) umma_commit(b_o);
        ++q;
      }
    }
  } else {
    // ---- softmax and output: key (then latent column) r of the tile ----
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const uint32_t lane_off = (uint32_t)(quarter * 32) << 16;
    const float sc = a.scale * LOG2E;
    uint8_t* my_p = base_ptr + cv.p + r * 128;
    int t = 0, q = 0;
    for (int w = blockIdx.x; w < total; w += gridDim.x) {
      const Unit u = unit_of(a, w, head_blocks);
      const int h0 = u.hb * NH, nh = min(NH, a.n_heads - h0);
      const size_t ih0 = (size_t)u.item * a.n_heads + h0;
      float l[NH];
#pragma unroll
      for (int h = 0; h < NH; ++h) l[h] = 0.f;
      bool ok = true;
      for (int j = 0; j < u.tiles; ++j, ++t) {
        ok = mbar_wait_bounded(b_s, t & 1);
        ok = !named_bar_or(1, 128, !ok);
        if (!ok) break;
        tc_fence_after();
        const bool seen = u.begin + j * KEYS + r < u.end;
        float wm[G];
        bool raise = j == 0;
        {
          uint32_t sv[NH];
          ld_heads<NH>(t_s + lane_off, sv);
          float v[NH];
#pragma unroll
          for (int h = 0; h < NH; ++h) v[h] = seen ? __uint_as_float(sv[h]) * sc : -INFINITY;
#pragma unroll
          for (int g = 0; g < G; ++g) wm[g] = reduce_columns<N1>(v + g * 32, lane, [](float x, float y) { return fmaxf(x, y); });
        }
        const int my_h = lane / (32 / N1);
#pragma unroll
        for (int g = 0; g < G; ++g) {
          if (j > 0) raise = raise || wm[g] > s_ref[my_h + g * 32] + RAISE;
          s_wmax[quarter][my_h + g * 32] = wm[g];
        }
        if (named_bar_or(1, 128, raise)) {
          const int h = threadIdx.x - 64;
          if (h < NH) {
            float mx = fmaxf(fmaxf(s_wmax[0][h], s_wmax[1][h]), fmaxf(s_wmax[2][h], s_wmax[3][h]));
            const float old = j > 0 ? s_ref[h] : -INFINITY;
            if (!(mx > old + RAISE)) mx = old;
            s_alpha[h] = j > 0 ? exp2f(old - mx) : 0.f;
            s_ref[h] = mx;
          }
          named_bar_sync(1, 128);
          if (j > 0) {
            // the scores of this tile were issued after the last product with P: O is complete
#pragma unroll
            for (int h = 0; h < NH; ++h) l[h] *= s_alpha[h];
            for (int d = 0; d < n_d; ++d) {
              uint32_t o[NH];
              ld_heads<NH>(t_o + d * NH + lane_off, o);
#pragma unroll
              for (int h = 0; h < NH; ++h) o[h] = __float_as_uint(__uint_as_float(o[h]) * s_alpha[h]);
              st_heads<NH>(t_o + d * NH + lane_off, o);
            }
            tmem_wait_st();
          }
        }
        {
          uint32_t sv[NH];
          ld_heads<NH>(t_s + lane_off, sv);
#pragma unroll
          for (int c = 0; c < NH / 8; ++c) {
            uint32_t pk[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int h = c * 8 + 2 * e;
              const float p0 = seen ? ex2_fast(fmaf(__uint_as_float(sv[h]), sc, -s_ref[h])) : 0.f;
              const float p1 = seen ? ex2_fast(fmaf(__uint_as_float(sv[h + 1]), sc, -s_ref[h + 1])) : 0.f;
              l[h] += p0;
              l[h + 1] += p1;
              pk[e] = pack2_prob(p0, p1, F16 ? 1 : 0);
            }
            *reinterpret_cast<uint4*>(my_p + ((c ^ (r & 7)) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
          }
        }
        fence_proxy_async_smem();
        tc_fence_before();
        mbar_arrive(b_p);
      }
      if (ok && u.tiles) {
        ok = mbar_wait_bounded(b_o, q & 1);
        ++q;
      }
      ok = !named_bar_or(1, 128, !ok);
      if (!ok) {
        arcb_set_error(a.err, ARCB_DEV_WAIT_TIMEOUT_ACC);
        break;
      }
      // denominators: over the lanes, then over the warps in a fixed order
#pragma unroll
      for (int g = 0; g < G; ++g) {
        const float s = reduce_columns<N1>(l + g * 32, lane, [](float x, float y) { return x + y; });
        s_l[quarter][lane / (32 / N1) + g * 32] = s;
      }
      named_bar_sync(1, 128);
      {
        const int h = threadIdx.x - 64;
        if (h < NH) {
          float lt = (s_l[0][h] + s_l[1][h]) + (s_l[2][h] + s_l[3][h]);
          float ref = u.tiles ? s_ref[h] : -INFINITY;
          if (a.n_splits > 1) {
            s_inv[h] = 1.f;
            if (h < nh) {
              float* rec = a.scratch + ((ih0 + h) * a.n_splits + u.split) * (a.kvp + 4);
              rec[a.kvp] = ref;
              rec[a.kvp + 1] = lt;
            }
          } else {
            float num = 1.f;
            if (a.sink && u.tiles && h < nh) {
              const float dlt = a.sink[h0 + h] * LOG2E - ref;
              if (dlt > 0.f) {      // bring both terms to the larger reference
                num = exp2f(-dlt);
                lt = lt * num + 1.f;
              } else {
                lt += exp2f(dlt);
              }
            }
            s_inv[h] = lt > 0.f ? num / lt : 0.f;
          }
        }
      }
      named_bar_sync(1, 128);
      tc_fence_after();
      for (int d = 0; d < n_d; ++d) {
        uint32_t o[NH];
        if (u.tiles) {
          ld_heads<NH>(t_o + d * NH + lane_off, o);
        } else {
#pragma unroll
          for (int h = 0; h < NH; ++h) o[h] = 0u;
        }
        const int col = d * 128 + r;
#pragma unroll
        for (int h = 0; h < NH; ++h) {
          if (h >= nh) break;
          const float v = __uint_as_float(o[h]) * s_inv[h];
          if (a.n_splits > 1) a.scratch[((ih0 + h) * a.n_splits + u.split) * (a.kvp + 4) + col] = v;
          else st_act(a.out, (ih0 + h) * a.kvp + col, v, F16 ? 1 : 0);
        }
      }
      tc_fence_before();
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(s_tmem, TMEM_COLS);
  }
}

template <int NH>
cudaError_t set_attr() {
  const int bytes = 227 * 1024 - STATIC_SMEM;
  cudaError_t e = cudaFuncSetAttribute(attn_latent_tc_kernel<NH, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) return e;
  return cudaFuncSetAttribute(attn_latent_tc_kernel<NH, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
}

template <int NH>
int launch(const AttnLatentArgs& a, cudaStream_t stream) {
  CUtensorMap tc, tl, tr;
  const int f16 = a.fmt == 1;
  const uint64_t qrows = (uint64_t)a.n_items * a.n_heads;
  int r = arcb_make_tmap_2d_16b(&tc, a.cache, (uint64_t)a.n_seqs * a.t_max, (uint64_t)(a.kvp + a.rotp), KEYS, 64, f16);
  if (!r) r = arcb_make_tmap_2d_16b(&tl, a.qlat, qrows, (uint64_t)a.kvp, NH, 64, f16);
  if (!r) r = arcb_make_tmap_2d_16b(&tr, a.q, qrows, (uint64_t)a.q_head, NH, 64, f16);
  if (r) return 1000 + r;
  const int slots = ring_slots(a.kvp, NH), hb = (a.n_heads + NH - 1) / NH;
  if (slots < a.kvp / 128) return -1;
  const long long total = (long long)a.n_items * a.n_splits * hb;
  if (total > 0x7fffffffLL) return -1;
  const int fmt = f16 ? 0 : 1;
  const uint32_t is = umma_idesc_f16(KEYS, NH, fmt, fmt, 0, 0), io = umma_idesc_f16(128, NH, fmt, fmt, 1, 1);
  const dim3 grid((unsigned)(total < 148 ? total : 148));
  const size_t smem = carve(a.kvp, NH, slots).total + 1024;
  const cudaError_t e = f16 ? arcb_launch(attn_latent_tc_kernel<NH, true>, grid, dim3(THREADS), smem, stream, tc, tl, tr, a, is, io, slots, hb, (int)total)
                            : arcb_launch(attn_latent_tc_kernel<NH, false>, grid, dim3(THREADS), smem, stream, tc, tl, tr, a, is, io, slots, hb, (int)total);
  arcb_count_launch(1);
  return (int)e;
}

}  // namespace

bool arcb_attn_latent_tc_supported(int kvp, int rotp, int fmt, int n_seqs, int t_max, float scale) {
  // the reference maxima follow the largest raw score, which needs a positive scale
  return fmt != 2 && scale > 0.f && kvp % 128 == 0 && kvp <= 512 && rotp == 64 && (long long)n_seqs * t_max < (1ll << 31) - 256;
}

int arcb_attn_latent_splits(int n_items, int n_heads, int kvp, int keys) {
  // one unit per SM at least, none shorter than two tiles
  const int nh = heads_of_block(n_heads, kvp);
  const long long units = (long long)n_items * ((n_heads + nh - 1) / nh);
  long long s = 148 / (units < 1 ? 1 : units);
  const long long most = (keys + 2 * KEYS - 1) / (2 * KEYS);
  if (keys > 0 && s > most) s = most;
  if (s > 32) s = 32;
  return s < 1 ? 1 : (int)s;
}

int arcb_attn_latent_init() {
  cudaError_t e;
  if ((e = set_attr<16>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<32>()) != cudaSuccess) return (int)e;
  if ((e = set_attr<64>()) != cudaSuccess) return (int)e;
  return 0;
}

int arcb_launch_attn_latent_tc(const AttnLatentArgs& a, cudaStream_t stream) {
  if (a.n_items <= 0) return 0;
  if (!arcb_attn_latent_tc_supported(a.kvp, a.rotp, a.fmt, a.n_seqs, a.t_max, a.scale) || a.q_off % 8 || a.q_head % 8) return -1;
  if (a.n_splits < 1 || (a.n_splits > 1 && !a.scratch)) return -1;
  const int nh = heads_of_block(a.n_heads, a.kvp);
  const int r = nh == 16 ? launch<16>(a, stream) : nh == 32 ? launch<32>(a, stream) : launch<64>(a, stream);
  if (r || a.n_splits == 1) return r;
  AttnGqaArgs c{};
  c.out = a.out; c.sink = a.sink; c.n_items = a.n_items; c.n_heads = a.n_heads; c.vdimp = a.kvp; c.n_splits = a.n_splits;
  c.scratch = a.scratch; c.fmt = a.fmt;
  return arcb_launch_attn_combine(c, stream);
}
