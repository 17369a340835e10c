// Causal prefill attention of grouped heads over the cache, on tcgen05 / TMEM; see attn_prefill_gqa.cu.
#pragma once
#include "common.cuh"

struct AttnPrefillGqaArgs {
  const void* q;               // 16-bit; row i, head h at q + i * q_pitch + q_col + h * dimp
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
  float scale;
  int act_f16;
  int* err;
};

bool arcb_attn_prefill_gqa_supported(int dimp, int vdimp, int n_seqs, int n_kv, int t_max, float scale);
int arcb_attn_prefill_gqa_init();
int arcb_launch_attn_prefill_gqa(const AttnPrefillGqaArgs& a, cudaStream_t stream);
void arcb_count_launch(long long n);
