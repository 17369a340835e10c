// Routing of tokens to experts, on the device without a host round trip:
//   route   : sigmoid of the router logits (fp32), the `top` largest scores of every row (the first of equal ones),
//             and the row's place among the tokens of each chosen expert
//   scatter : slots of every expert (padded to whole tiles of the grouped product), expert of every tile, rows of xn
//             in slot order, slot and weight of every (row, choice)
// Slots of one expert are filled in no particular order: a row's result does not depend on its slot.
#include "launch.cuh"
#include "moe.cuh"

namespace {

// The chosen experts of a row by one warp; lane i holds the scores of experts i, i + 32, ... in s.  Lane k returns
// the k-th choice.
template <int PER_LANE>
__device__ __forceinline__ int choose(const MoeArgs& a, int lane, float (&s)[PER_LANE], float& my_w) {
  int my_e = 0;
  my_w = 0.f;
  for (int k = 0; k < a.top; ++k) {
    // scores lie in [0, 1]: their bits order like the numbers, and ~e prefers the first of equal ones
    unsigned long long best = 0;
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) {
      if (s[i] >= 0.f) {
        const unsigned long long key = ((unsigned long long)(__float_as_uint(s[i]) + 1u) << 32) | (uint32_t)~(lane + 32 * i);
        best = key > best ? key : best;
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const unsigned long long t = __shfl_xor_sync(0xffffffffu, best, o);
      best = t > best ? t : best;
    }
    const int e = best ? (int)~(uint32_t)best : k;      // no score is a number: any expert, weight 0
    if (lane == k) {
      my_e = e;
      my_w = best ? __uint_as_float((uint32_t)(best >> 32) - 1u) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i)
      if (lane + 32 * i == e) s[i] = -1.f;
  }
  return my_e;
}

__device__ __forceinline__ float score(float z) { return 1.f / (1.f + expf(-z)); }

// One warp per row and turn; ranks are counted within the CTA first, so that an expert's counter is touched once per CTA.
constexpr int ROUTE_ROWS = 32;
template <int PER_LANE>
__global__ void __launch_bounds__(128)
moe_route_kernel(MoeArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ int s_count[MOE_MAX_EXPERTS], s_base[MOE_MAX_EXPERTS];
  const int row0 = blockIdx.x * ROUTE_ROWS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int e = threadIdx.x; e < a.experts; e += 128) s_count[e] = 0;
  __syncthreads();
  int my_e[ROUTE_ROWS / 4], my_r[ROUTE_ROWS / 4];
#pragma unroll
  for (int t = 0; t < ROUTE_ROWS / 4; ++t) {
    const int row = row0 + t * 4 + warp;
    my_e[t] = my_r[t] = 0;
    if (row >= a.rows) continue;
    float s[PER_LANE];
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) {
      const int e = lane + 32 * i;
      s[i] = e < a.experts ? score(a.z[(size_t)row * a.z_pitch + e]) : -1.f;
    }
    float w;
    my_e[t] = choose<PER_LANE>(a, lane, s, w);
    if (lane < a.top) {
      a.expert[(size_t)row * a.top + lane] = my_e[t];
      a.weight[(size_t)row * a.top + lane] = w;
      my_r[t] = atomicAdd(s_count + my_e[t], 1);
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < a.experts; e += 128) s_base[e] = s_count[e] ? atomicAdd(a.count + e, s_count[e]) : 0;
  __syncthreads();
#pragma unroll
  for (int t = 0; t < ROUTE_ROWS / 4; ++t) {
    const int row = row0 + t * 4 + warp;
    if (row < a.rows && lane < a.top) a.rank[(size_t)row * a.top + lane] = s_base[my_e[t]] + my_r[t];
  }
}

// One CTA of eight warps per ROUTER_ROWS rows, which also multiplies the rows with the router (16-bit formats).
constexpr int ROUTER_WARPS = 8, ROUTER_ROWS = 2;
template <int PER_LANE>
__global__ void __launch_bounds__(ROUTER_WARPS * 32)
moe_router_kernel(MoeArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float s_z[ROUTER_ROWS][MOE_MAX_EXPERTS];
  const int row0 = blockIdx.x * ROUTER_ROWS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = a.pitch / 8;                             // 8 columns a load
  const uint4* x[ROUTER_ROWS];
#pragma unroll
  for (int r = 0; r < ROUTER_ROWS; ++r)
    x[r] = reinterpret_cast<const uint4*>(reinterpret_cast<const uint16_t*>(a.xn) + (size_t)min(row0 + r, a.rows - 1) * a.pitch);
  for (int e0 = warp * 4; e0 < a.experts; e0 += ROUTER_WARPS * 4) {
    float d[ROUTER_ROWS][4] = {};
    const uint4* w = reinterpret_cast<const uint4*>(reinterpret_cast<const uint16_t*>(a.w_router) + (size_t)e0 * a.pitch);
#pragma unroll 2
    for (int i = lane; i < n; i += 32) {                 // rows behind the last expert are zero
      uint4 wv[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) wv[e] = __ldg(w + (size_t)e * n + i);
#pragma unroll
      for (int r = 0; r < ROUTER_ROWS; ++r) {
        const uint4 xv = x[r][i];
        const uint32_t xr[4] = {xv.x, xv.y, xv.z, xv.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 p = unpack2_act(xr[j], a.fmt);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const uint32_t wr[4] = {wv[e].x, wv[e].y, wv[e].z, wv[e].w};
            const float2 q = unpack2_act(wr[j], a.fmt);
            d[r][e] = fmaf(p.x, q.x, d[r][e]);
            d[r][e] = fmaf(p.y, q.y, d[r][e]);
          }
        }
      }
    }
#pragma unroll
    for (int r = 0; r < ROUTER_ROWS; ++r)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        d[r][e] = warp_sum(d[r][e]);
        if (lane == 0 && e0 + e < a.experts) s_z[r][e0 + e] = d[r][e];
      }
  }
  __syncthreads();
  const int row = row0 + warp;
  if (warp >= ROUTER_ROWS || row >= a.rows) return;
  float s[PER_LANE];
#pragma unroll
  for (int i = 0; i < PER_LANE; ++i) {
    const int e = lane + 32 * i;
    s[i] = e < a.experts ? score(s_z[warp][e]) : -1.f;
  }
  float w;
  const int e = choose<PER_LANE>(a, lane, s, w);
  if (lane < a.top) {
    const size_t at = (size_t)row * a.top + lane;
    a.expert[at] = e;
    a.weight[at] = w;
    a.rank[at] = atomicAdd(a.count + e, 1);
  }
}

// One CTA per row.  Every CTA takes the running sum over the experts' padded counts for itself; the first one also
// lists the tiles and clears the padding slots' weights.
constexpr int SCATTER_THREADS = 128;
__global__ void __launch_bounds__(SCATTER_THREADS)
moe_scatter_kernel(MoeArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ int s_first[MOE_MAX_EXPERTS + 1];
  __shared__ int s_slot[MOE_MAX_TOP];
  __shared__ int s_warp[2 * SCATTER_THREADS / 32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  int incl[2], padded[2];                                // experts tid and tid + 128
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int e = tid + i * SCATTER_THREADS;
    padded[i] = e < a.experts ? (a.count[e] + a.gran - 1) / a.gran * a.gran : 0;
    int v = padded[i];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int t = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= o) v += t;
    }
    incl[i] = v;
    if (lane == 31) s_warp[i * (SCATTER_THREADS / 32) + warp] = v;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    int before = 0;
    for (int j = 0; j < i * (SCATTER_THREADS / 32) + warp; ++j) before += s_warp[j];
    const int e = tid + i * SCATTER_THREADS;
    s_first[e] = before + incl[i] - padded[i];
    if (e == MOE_MAX_EXPERTS - 1) s_first[MOE_MAX_EXPERTS] = before + incl[i];
  }
  __syncthreads();
  const int row = blockIdx.x;
  if (row == 0) {
    for (int e = warp; e < a.experts; e += SCATTER_THREADS / 32) {
      const int first = s_first[e], n = a.count[e], end = (n + a.gran - 1) / a.gran * a.gran;
      for (int t = lane * 128; t < end; t += 32 * 128) a.tile_expert[(first + t) >> 7] = e;
      for (int i = n + lane; i < end; i += 32) a.slot_weight[first + i] = 0.f;
    }
    if (tid == 0) *a.n_tiles = s_first[MOE_MAX_EXPERTS] >> 7;
  }
  if (tid < a.top) {
    const size_t at = (size_t)row * a.top + tid;
    const int slot = s_first[a.expert[at]] + a.rank[at];
    s_slot[tid] = slot;
    a.slot[at] = slot;
    a.slot_weight[slot] = a.weight[at];
  }
  __syncthreads();
  const size_t bytes = (size_t)a.pitch * act_bytes(a.fmt);
  const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const uint8_t*>(a.xn) + row * bytes);
  for (int i = tid; i < (int)(bytes / 16); i += SCATTER_THREADS) {
    const uint4 v = src[i];
    for (int k = 0; k < a.top; ++k) reinterpret_cast<uint4*>(reinterpret_cast<uint8_t*>(a.xs) + s_slot[k] * bytes)[i] = v;
  }
}

}  // namespace

int arcb_moe_max_slots(int rows, int experts, int top, int gran) {
  // every expert with a token wastes less than gran slots
  const long long n = (long long)rows * top, used = n < experts ? n : experts;
  const long long s = n + used * (gran - 1);
  return (int)((s + gran - 1) / gran * gran);
}

bool arcb_moe_router_inside(int rows, int experts, int pitch, int fmt) {
  return fmt != 2 && (long long)rows * experts * pitch <= 32ll << 20;     // 64 MB of weights through the L2 cache
}

int arcb_launch_moe_route(const MoeArgs& a, cudaStream_t stream) {
  if (a.rows <= 0) return 0;
  if (a.experts > MOE_MAX_EXPERTS || a.top > MOE_MAX_TOP || a.top > a.experts || a.top < 1 || a.pitch % 8) return -1;
  if (a.max_slots < arcb_moe_max_slots(a.rows, a.experts, a.top, a.gran)) return -1;
  auto go = [&](auto route, auto router) {
    return a.z ? arcb_launch(route, dim3((a.rows + ROUTE_ROWS - 1) / ROUTE_ROWS), dim3(128), 0, stream, a)
               : arcb_launch(router, dim3((a.rows + ROUTER_ROWS - 1) / ROUTER_ROWS), dim3(ROUTER_WARPS * 32), 0, stream, a);
  };
  cudaError_t e = a.experts <= 32    ? go(moe_route_kernel<1>, moe_router_kernel<1>)
                  : a.experts <= 64  ? go(moe_route_kernel<2>, moe_router_kernel<2>)
                  : a.experts <= 128 ? go(moe_route_kernel<4>, moe_router_kernel<4>)
                                     : go(moe_route_kernel<8>, moe_router_kernel<8>);
  if (e != cudaSuccess) return (int)e;
  e = arcb_launch(moe_scatter_kernel, dim3(a.rows), dim3(SCATTER_THREADS), 0, stream, a);
  arcb_count_launch(2);
  return (int)e;
}
