// Causal prefill attention on tcgen05 / TMEM, over the cache of grouped heads or over keys and values expanded from
// cached latents; see attn_prefill_gqa.cu.
#pragma once
#include "common.cuh"

struct AttnPrefillGqaArgs {
  const void* q;               // 16-bit; row i, head h at q + i * q_pitch + q_col + h * (dimp + rotp)
  long long q_pitch;
  int q_col;
  const void* k;               // [n_seqs][G][t_max][dimp], the same 16-bit format
  const void* v;               // [n_seqs][G][t_max][vdimp]
  const void* gate;            // optional sigmoid gates, row i, head h at gate + i * gate_pitch + h * vdimp
  long long gate_pitch;
  void* out;                   // [n_rows][H][vdimp]
  const int* seq;              // [n_rows] cache row
  const int* kv_count;         // [n_rows] visible keys
  const int* qblock_row0;      // query blocks of 1..256 consecutive rows of one sequence
  const int* qblock_rows;
  const float* sink;           // optional [H]
  int n_qblocks, n_rows, n_heads, n_kv, dimp, vdimp, t_max, n_seqs;
  int window;                  // keys [count - window, count) are visible, 0: all [0, count)
  // Expanded keys and values (kv0 set): key / value of position p and head h are columns [h * dimp, ...) and
  // [v_col + h * vdimp, ...) of row kv0[block] + p of a matrix with kv_pitch columns; the last rotp dimensions of
  // every head's key are row (seq * rot_panels + rot_panel) * t_max + p of k_rot (64 columns).
  const int* kv0;              // [n_qblocks]
  long long kv_rows, kv_pitch;
  int v_col;
  const void* k_rot;
  int rotp, rot_panels, rot_panel;
  float scale;
  int act_f16;
  int* err;
};

bool arcb_attn_prefill_gqa_supported(int dimp, int vdimp, int n_seqs, int n_kv, int t_max, float scale);
bool arcb_attn_prefill_latent_supported(int dimp, int rotp, int vdimp, int panels, int n_seqs, int t_max, float scale);
int arcb_attn_prefill_gqa_init();
int arcb_launch_attn_prefill_gqa(const AttnPrefillGqaArgs& a, cudaStream_t stream);
void arcb_count_launch(long long n);
