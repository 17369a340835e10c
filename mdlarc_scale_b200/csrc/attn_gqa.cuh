// Streaming attention of one query row over a cached prefix with grouped heads: arguments and launcher
// (attn_gqa.cu); the kernel template is in attn_gqa_impl.cuh.
#pragma once
#include "common.cuh"

struct AttnGqaArgs {
  const void* q;              // row i, head h at q + i * q_pitch + h * dimp (activation format)
  long long q_pitch;
  const void* k;              // [n_seqs][G][t_max][dimp] activation format
  const void* v;              // [n_seqs][G][t_max][vdimp]
  const void* gate;           // optional sigmoid gates: row i, head h at gate + i * gate_pitch + h * vdimp
  long long gate_pitch;
  void* out;                  // [n_items][H][vdimp] activation format
  const int* item_seq;        // [n_items] cache row, null = item index
  const int* item_len;        // [n_items] keys [0, len) are attended,
  int window;                 //   or the last `window` of them when window > 0
  const float* sink;          // optional [H]: exp(sink) joins the softmax denominator
  int n_items, n_heads, n_kv, dimp, vdimp, t_max, n_seqs, n_splits;
  float scale;
  float* scratch;             // n_items * H * n_splits * (vdimp + 4) floats when n_splits > 1
  int fmt;
  int* err;
  // filled by the launcher
  int rep, tiles, tile_rows;  // query heads per key/value head, and how they are tiled
};

int arcb_launch_attn_gqa(AttnGqaArgs a, cudaStream_t stream);
// merges the splits in a.scratch ([item][head][split][vdimp + 4]: sums, reference maximum in log2 units, denominator)
int arcb_launch_attn_combine(const AttnGqaArgs& a, cudaStream_t stream);
// splits of a decode launch (upper bound used for the scratch when t_max is 0)
int arcb_attn_gqa_splits(int n_items, int n_kv, int rep, int t_max);
void arcb_count_launch(long long n);

// one translation unit per activation format
cudaError_t arcb_attn_gqa_dispatch_f16(const AttnGqaArgs& a, dim3 grid, cudaStream_t stream);
cudaError_t arcb_attn_gqa_dispatch_bf16(const AttnGqaArgs& a, dim3 grid, cudaStream_t stream);
cudaError_t arcb_attn_gqa_dispatch_f32(const AttnGqaArgs& a, dim3 grid, cudaStream_t stream);
