// Matrix-memory recurrence (mLSTM): arguments and launchers; see mlstm.cu.
//
// Per head, with log gates i_t and f_t, a running stabiliser m and state S [dim][vdim], n [dim]:
//   m_t = max(f_t + m_{t-1}, i_t)
//   S_t = exp(f_t + m_{t-1} - m_t) S_{t-1} + exp(i_t - m_t) k_t v_t^T          (n alike with k_t alone)
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
// followed by the head's RMS norm, the gain and the output gate.
#pragma once
#include "common.cuh"

// capped log gates of the recurrence from the biased pre-activation
__device__ __forceinline__ float gate_log(float x, float cap, bool forget) {
  const float z = cap * tanhf(x / cap);
  if (!forget) return z;
  return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));   // log sigmoid
}

struct MlstmArgs {
  const void* proj;          // [rows][pitch] activation format: q, k, v and sigmoid output gates
  long long pitch;
  int off_q, off_k, off_v, off_g;
  const float* gates;        // [rows][2 H] biased pre-activations of the input gates, then of the forget gates
  float gate_cap;
  const float* norm_w;       // [H][vdimp]
  void* out;                 // [rows][H][vdimp] activation format
  float* S;                  // [n_seqs][H][dim][vdimp]
  float* n;                  // [n_seqs][H][dimp]
  float* m;                  // [n_seqs][H]
  int H, dim, dimp, vdim, vdimp, n_seqs, fmt;
  int n_rows;                // rows of proj
  float eps;
  // segments of consecutive rows; null seg_seq: row b belongs to sequence b (one row each) at position
  // pos[b], < 0 = held
  const int* seg_row0; const int* seg_rows; const int* seg_seq; const int* seg_pos0;
  const int* pos;
  int n_segs;
  int* err;
};

bool arcb_mlstm_chunk_supported(int dimp, int vdimp, int fmt);
int arcb_mlstm_chunk_init();
int arcb_launch_mlstm_chunk(const MlstmArgs& a, cudaStream_t stream);
int arcb_launch_mlstm_step(const MlstmArgs& a, cudaStream_t stream);
void arcb_count_launch(long long n);
