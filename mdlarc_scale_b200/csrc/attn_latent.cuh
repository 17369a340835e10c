// Attention of one query row per item over cached latents: arguments and launchers; see attn_latent.cu (tensor cores)
// and attn_latent_stream.cu (any size, any format).
#pragma once
#include "common.cuh"

// The queries are already in the latent space: head h of item i scores position p with
//   (qlat[i][h] . c[p] + qrot[i][h] . r[p]) * scale,   cached row p = [c (kvp columns) | r (rotp columns)],
// and the output row is the weighted sum of c.  A sequence's rows are cut into panels of 64 columns, each panel's rows
// side by side: whatever reads 64 columns of many rows then reads one piece of memory.
struct AttnLatentArgs {
  const void* qlat;          // [n_items][H][kvp] activation format
  const void* q;             // rotated part: row i, head h at q + i * H * q_head + h * q_head + q_off
  int q_head, q_off;
  const void* cache;         // [n_seqs][(kvp + rotp) / 64][t_max][64]
  void* out;                 // [n_items][H][kvp]
  const int* item_seq;       // [n_items] cache row, null = item index
  const int* item_len;       // [n_items] positions [0, len) are cached up to and with the query's own
  const float* sink;         // optional [H]: exp(sink) joins the softmax denominator
  int n_items, n_heads, kvp, rotp, t_max, n_seqs, n_splits;
  int window;                // positions [len - window, len) are visible, 0: all
  float scale;
  float* scratch;            // n_items * H * n_splits * (kvp + 4) floats when n_splits > 1
  int fmt;
  int* err;
};

bool arcb_attn_latent_tc_supported(int kvp, int rotp, int fmt, int n_seqs, int t_max, float scale);
int arcb_attn_latent_splits(int n_items, int n_heads, int kvp, int keys);
int arcb_attn_latent_init();
int arcb_launch_attn_latent_tc(const AttnLatentArgs& a, cudaStream_t stream);
int arcb_launch_attn_latent_stream(const AttnLatentArgs& a, cudaStream_t stream);
void arcb_count_launch(long long n);
