// Routing of tokens to experts, on the device without a host round trip:
//   route   : sigmoid of the router logits (fp32), the `top` largest scores of every row (the first of equal ones),
//             and the row's place among the tokens of each chosen expert
//   plan    : slots of every expert (padded to whole tiles of the grouped product), expert of every tile
//   scatter : rows of xn in slot order, slot and weight of every (row, choice)
// Slots of one expert are filled in no particular order: a row's result does not depend on its slot.
#include "launch.cuh"
#include "moe.cuh"

namespace {

constexpr int PER_LANE = MOE_MAX_EXPERTS / 32;
constexpr int PLAN_THREADS = 256;
static_assert(PLAN_THREADS == MOE_MAX_EXPERTS, "one thread of the plan per expert");

// One warp per row; lane i holds the scores of experts i, i + 32, ...
__global__ void __launch_bounds__(128)
moe_route_kernel(MoeArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= a.rows) return;
  float s[PER_LANE];
#pragma unroll
  for (int i = 0; i < PER_LANE; ++i) {
    const int e = lane + 32 * i;
    s[i] = e < a.experts ? 1.f / (1.f + expf(-a.z[(size_t)row * a.z_pitch + e])) : -1.f;
  }
  int my_e = 0;
  float my_w = 0.f;
  for (int k = 0; k < a.top; ++k) {
    // scores lie in [0, 1]: their bits order like the numbers, and ~e prefers the first of equal ones
    unsigned long long best = 0;
#pragma unroll
    for (int i = 0; i < PER_LANE; ++i) {
      const int e = lane + 32 * i;
      if (s[i] >= 0.f) {
        const unsigned long long key = ((unsigned long long)(__float_as_uint(s[i]) + 1u) << 32) | (uint32_t)~e;
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
  if (lane < a.top) {
    const size_t at = (size_t)row * a.top + lane;
    a.expert[at] = my_e;
    a.weight[at] = my_w;
    a.rank[at] = atomicAdd(a.count + my_e, 1);
  }
}

// One CTA, one thread per expert.
__global__ void __launch_bounds__(PLAN_THREADS)
moe_plan_kernel(MoeArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ int scan[PLAN_THREADS];
  const int e = threadIdx.x;
  const int n = e < a.experts ? a.count[e] : 0;
  const int padded = (n + a.gran - 1) / a.gran * a.gran;
  scan[e] = padded;
  __syncthreads();
#pragma unroll
  for (int o = 1; o < PLAN_THREADS; o <<= 1) {
    const int v = e >= o ? scan[e - o] : 0;
    __syncthreads();
    scan[e] += v;
    __syncthreads();
  }
  const int first = scan[e] - padded;
  if (e < a.experts) {
    a.offset[e] = first;
    a.count[e] = 0;
    for (int t = 0; t < padded; t += 128) a.tile_expert[(first + t) >> 7] = e;
    for (int i = n; i < padded; ++i) a.slot_weight[first + i] = 0.f;
  }
  if (e == PLAN_THREADS - 1) *a.n_tiles = scan[e] >> 7;
}

// One warp per (row, choice).
__global__ void __launch_bounds__(128)
moe_scatter_kernel(MoeArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const long long w = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (w >= (long long)a.rows * a.top) return;
  const int row = (int)(w / a.top);
  const int slot = a.offset[a.expert[w]] + a.rank[w];
  if (lane == 0) {
    a.slot[w] = slot;
    a.slot_weight[slot] = a.weight[w];
  }
  const size_t bytes = (size_t)a.pitch * act_bytes(a.fmt);
  const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const uint8_t*>(a.xn) + row * bytes);
  uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<uint8_t*>(a.xs) + slot * bytes);
  for (int i = lane; i < (int)(bytes / 16); i += 32) dst[i] = src[i];
}

}  // namespace

int arcb_moe_max_slots(int rows, int experts, int top, int gran) {
  // every expert with a token wastes less than gran slots
  const long long n = (long long)rows * top, used = n < experts ? n : experts;
  const long long s = n + used * (gran - 1);
  return (int)((s + gran - 1) / gran * gran);
}

int arcb_launch_moe_route(const MoeArgs& a, cudaStream_t stream) {
  if (a.rows <= 0) return 0;
  if (a.experts > MOE_MAX_EXPERTS || a.top > MOE_MAX_TOP || a.top > a.experts || a.top < 1) return -1;
  if (a.max_slots < arcb_moe_max_slots(a.rows, a.experts, a.top, a.gran)) return -1;
  cudaError_t e = arcb_launch(moe_route_kernel, dim3((a.rows + 3) / 4), dim3(128), 0, stream, a);
  if (e != cudaSuccess) return (int)e;
  e = arcb_launch(moe_plan_kernel, dim3(1), dim3(PLAN_THREADS), 0, stream, a);
  if (e != cudaSuccess) return (int)e;
  const long long n = ((long long)a.rows * a.top + 3) / 4;
  e = arcb_launch(moe_scatter_kernel, dim3((unsigned)n), dim3(128), 0, stream, a);
  arcb_count_launch(3);
  return (int)e;
}
