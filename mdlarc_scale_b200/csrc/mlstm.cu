// Token-by-token form of the matrix-memory recurrence: the decode step, and prefill where the chunkwise
// kernel does not apply.
//
// One CTA owns one (segment, head) and keeps the whole fp32 state in registers while it walks the
// segment's tokens: thread (rg, c4) holds rows rg, rg + RG, ... of four neighbouring value columns.  A
// decode step reads and writes the state once, 16 bytes a lane and contiguous across the warp, with all
// of a thread's loads in flight together; nothing else of the step is large, so the launch is bound by
// that traffic.  The head's RMS norm, gain and output gate are applied before the row leaves.
#include "launch.cuh"
#include "mlstm.cuh"

namespace {

template <int DMAX, int VP>
struct MlstmCfg {
  static constexpr int NT = (DMAX * VP / 64 > 256) ? DMAX * VP / 64 : 256;
  static constexpr int C4 = VP / 4;          // threads across the value columns
  static constexpr int RG = NT / C4;         // row groups
  static constexpr int RPT = DMAX / RG;      // rows per thread
};

template <int DMAX, int VP>
__global__ void __launch_bounds__(MlstmCfg<DMAX, VP>::NT)
mlstm_step_kernel(MlstmArgs a) {
  using C = MlstmCfg<DMAX, VP>;
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float s_q[DMAX], s_k[DMAX];
  __shared__ __align__(16) float s_red[C::RG][VP];
  __shared__ float s_nq[C::NT / 32], s_ss[C::NT / 32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x, sg = blockIdx.y;
  int row0, rows, seq, pos0;
  if (a.seg_seq) {
    row0 = a.seg_row0[sg]; rows = a.seg_rows[sg]; seq = a.seg_seq[sg]; pos0 = a.seg_pos0[sg];
  } else {
    row0 = sg; seq = sg; pos0 = a.pos[sg]; rows = pos0 < 0 ? 0 : 1;
  }
  if (seq < 0 || seq >= a.n_seqs) {
    if (tid == 0) arcb_set_error(a.err, ARCB_DEV_BAD_INDEX);
    rows = 0;
  }
  if (rows <= 0) {
    // a held row still feeds the next product: give it zeros
    if (!a.seg_seq && tid < VP) st_act(a.out, ((size_t)row0 * a.H + h) * VP + tid, 0.f, a.fmt);
    return;
  }
  const int c4 = tid % C::C4, rg = tid / C::C4;
  float* Sg = a.S + ((size_t)seq * a.H + h) * a.dim * VP;
  float* ng = a.n + ((size_t)seq * a.H + h) * a.dimp;
  float* mg = a.m + (size_t)seq * a.H + h;

  float4 S[C::RPT];
  float n = 0.f, m = 0.f;
  const bool fresh = pos0 == 0;
#pragma unroll
  for (int j = 0; j < C::RPT; ++j) {
    const int r = rg + j * C::RG;
    S[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!fresh && r < a.dim) S[j] = *reinterpret_cast<const float4*>(Sg + (size_t)r * VP + c4 * 4);
  }
  if (!fresh) {
    if (tid < a.dim) n = ng[tid];
    m = *mg;
  }
  const float inv_v = 1.f / (float)a.vdim;
  for (int t = 0; t < rows; ++t) {
    const int row = row0 + t;
    const size_t base = (size_t)row * a.pitch;
    if (tid < DMAX) {
      s_q[tid] = tid < a.dim ? ld_act(a.proj, base + a.off_q + (size_t)h * a.dimp + tid, a.fmt) : 0.f;
      s_k[tid] = tid < a.dim ? ld_act(a.proj, base + a.off_k + (size_t)h * a.dimp + tid, a.fmt) : 0.f;
    }
    const float4 v = ld_act4(a.proj, base + a.off_v + (size_t)h * VP + c4 * 4, a.fmt);
    const float gi = gate_log(a.gates[(size_t)row * 2 * a.H + h], a.gate_cap, false);
    const float gf = gate_log(a.gates[(size_t)row * 2 * a.H + a.H + h], a.gate_cap, true);
    const float m_new = fmaxf(gf + m, gi);
    const float keep = expf(gf + m - m_new), add = expf(gi - m_new);
    m = m_new;
    __syncthreads();
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < C::RPT; ++j) {
      const int r = rg + j * C::RG;
      const float kk = add * s_k[r], qq = s_q[r];
      S[j].x = fmaf(kk, v.x, keep * S[j].x);
      S[j].y = fmaf(kk, v.y, keep * S[j].y);
      S[j].z = fmaf(kk, v.z, keep * S[j].z);
      S[j].w = fmaf(kk, v.w, keep * S[j].w);
      acc.x = fmaf(S[j].x, qq, acc.x);
      acc.y = fmaf(S[j].y, qq, acc.y);
      acc.z = fmaf(S[j].z, qq, acc.z);
      acc.w = fmaf(S[j].w, qq, acc.w);
    }
    *reinterpret_cast<float4*>(&s_red[rg][c4 * 4]) = acc;
    float nq = 0.f;
    if (tid < DMAX) {
      n = fmaf(add, s_k[tid], keep * n);
      nq = n * s_q[tid];
    }
    if (tid < ((DMAX + 31) & ~31)) {
      nq = warp_sum(nq);
      if (lane == 0) s_nq[warp] = nq;
    }
    __syncthreads();
    float o = 0.f;
    if (tid < VP) {
#pragma unroll
      for (int j = 0; j < C::RG; ++j) o += s_red[j][tid];
      float dot = 0.f;
#pragma unroll
      for (int j = 0; j < (DMAX + 31) / 32; ++j) dot += s_nq[j];
      o /= fmaxf(fabsf(dot), expf(-m)) + 1e-6f;
      const float ss = warp_sum(o * o);     // padding columns are exactly zero
      if (lane == 0) s_ss[warp] = ss;
    }
    __syncthreads();
    if (tid < VP) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < VP / 32; ++j) ss += s_ss[j];
      o *= 1.f / sqrtf(ss * inv_v + a.eps);
      o *= a.norm_w[(size_t)h * VP + tid] * ld_act(a.proj, base + a.off_g + (size_t)h * VP + tid, a.fmt);
      st_act(a.out, ((size_t)row * a.H + h) * VP + tid, o, a.fmt);
    }
  }
#pragma unroll
  for (int j = 0; j < C::RPT; ++j) {
    const int r = rg + j * C::RG;
    if (r < a.dim) *reinterpret_cast<float4*>(Sg + (size_t)r * VP + c4 * 4) = S[j];
  }
  if (tid < a.dim) ng[tid] = n;
  if (tid == 0) *mg = m;
}

template <int DMAX, int VP>
cudaError_t launch_step(const MlstmArgs& a, cudaStream_t stream) {
  return arcb_launch(mlstm_step_kernel<DMAX, VP>, dim3(a.H, a.n_segs), dim3(MlstmCfg<DMAX, VP>::NT), 0, stream, a);
}

}  // namespace

int arcb_launch_mlstm_step(const MlstmArgs& a, cudaStream_t stream) {
  if (a.n_segs <= 0) return 0;
  if (a.n_segs > 65535) return -1;
  cudaError_t e = cudaErrorInvalidValue;
  switch (a.dimp * 1000 + a.vdimp) {
    case 64064: e = launch_step<64, 64>(a, stream); break;
    case 64128: e = launch_step<64, 128>(a, stream); break;
    case 64256: e = launch_step<64, 256>(a, stream); break;
    case 128064: e = launch_step<128, 64>(a, stream); break;
    case 128128: e = launch_step<128, 128>(a, stream); break;
    case 128256: e = launch_step<128, 256>(a, stream); break;
    case 256064: e = launch_step<256, 64>(a, stream); break;
    case 256128: e = launch_step<256, 128>(a, stream); break;
    case 256256: e = launch_step<256, 256>(a, stream); break;
  }
  arcb_count_launch(1);
  return (int)e;
}
