// Row-wise kernels of layered models (embedding, norms, unfused projections, token picking) and their
// argument blocks; see layerops.cu.
#pragma once
#include "epilogue.cuh"

// Device-resident state of the decode loop of a layered session (arrays indexed by cache row).
struct StepState {
  int n_seqs, t_max, max_new, stop_on_end, end_token;
  int* cur_len;        // positions cached
  int* len0;           // cur_len when the sequence was armed
  int* cur_tok;        // token the next step feeds
  int* active;         // 1: the next step advances this sequence
  int* pos;            // [B] position (= cache slot) of the fed token, -1: held (written by step_begin)
  int* kv_len;         // [B] keys the step attends to, 0: held
  int* finished;       // [B]
  int* n_finished;
  int* out_tokens;     // [B][max_new]
  const int* forced;   // optional [B][max_new]
  float* step_logits;  // optional [B][max_new][vocab]
  float temperature;
  int top_k;
  unsigned long long sample_seed;
  const int* sample_stream;
  int* err;
};

struct LmEmbedArgs {
  int rows, width, pitch, vocab, fmt;
  const int* token_ids;    // [rows]; null in step_begin
  const float* embed;      // [vocab][pitch]
  float alpha;             // x leaves multiplied by the residual factor of the first sublayer
  float* x;                // [rows][pitch]
  void* xn;                // [rows][pitch] activation format, null: not written
  int* zero;               // optional counters the pass starts from
  int n_zero;
};

// y = norm(x) * w; xn gets y in the activation format, and x (optional) y * x_scale.
struct LmNormArgs {
  int kind;                // ARCB_NORM_*
  int rows, width, pitch, fmt;
  float eps, x_scale;
  float* x;                // [.][pitch]
  const float* w;          // [pitch]
  void* xn;                // [rows][pitch]
  int write_x;
  const int* row_index;    // optional gather of rows of x (write_x 0)
  float* dense;            // optional [rows][width]: y, without padding
};

// Sandwich norms, one sublayer to the next: x += norm(y) * w_out, then xn = norm(x) * w_in in the activation format.
// y is the sum of a fp32 row and of `top` rows of an expert product.
struct SandwichArgs {
  int rows, width, pitch, fmt, top;
  float eps;
  float* x;                // [rows][pitch]
  const float* y;          // [rows][pitch], null: zero
  const void* ye;          // activation format, rows slot[row * top + k]; null: none
  const int* slot;
  const float* w_out;      // [pitch]
  const float* w_in;       // [pitch], null: no norm behind the sum
  void* xn;                // [rows][pitch]
  float* dense;            // optional [rows][width]: x after the sum, without padding
  const float* embed;      // optional [vocab][pitch]: the row's embedding joins x after that
  const int* tokens;       // [rows]
  int vocab;
};

// Latent projections in fp32 -> normed query latent, and the cached row: normed latent and rotated key part.
struct LatentPrepArgs {
  int rows, pitch;         // proj [rows][pitch]: query latent at 0, latent at off_c, rotated part at off_r
  int q_rank, q_rankp, kv_rank, kv_rankp, rot_dim, rotp, off_c, off_r;
  const float* proj;
  const float* q_norm;     // [q_rankp]
  const float* kv_norm;    // [kv_rankp]
  float eps;
  const float2* rot;       // [t_max][rotp / 2] (cos, sin), null: nothing turns
  void* cq;                // [rows][q_rankp]
  void* cache;             // [n_seqs][(kv_rankp + rotp) / 64][t_max][64]
  const int* pos;          // [rows], negative: the row stores nothing
  const int* seq;          // [rows] cache row, null: row index
  int t_max, n_seqs, fmt;
  int* err;
};

enum : int { PICK_PLAIN = 0, PICK_FIRST = 1, PICK_DECODE = 2 };

struct PickArgs {
  int mode, rows, vocab, pitch;
  float* logits;           // [rows][pitch] raw, scaled in place
  float scale;
  float* out;              // optional [rows][vocab]
  const int* first_seq;    // PICK_FIRST
  const int* prompt_len;
};

int arcb_launch_lm_embed(const LmEmbedArgs& a, cudaStream_t stream);
int arcb_launch_step_begin(const StepState& st, const LmEmbedArgs& a, cudaStream_t stream);
int arcb_launch_lm_norm(const LmNormArgs& a, cudaStream_t stream);
int arcb_launch_sandwich_norm(const SandwichArgs& a, cudaStream_t stream);
int arcb_launch_latent_prep(const LatentPrepArgs& a, cudaStream_t stream);
// table[p][i] = (cos, sin)(p * base^(-2 i / dims)), i < dims / 2, and (1, 0) for i from there to pairs - 1
int arcb_launch_rot_table(float2* table, int t_max, int pairs, int dims, double base, cudaStream_t stream);
int arcb_launch_proj_prep(const ProjArgs& a, const float* proj, cudaStream_t stream);
int arcb_launch_pick(const PickArgs& a, const StepState& st, cudaStream_t stream);
int arcb_launch_seg_commit(const StepState& st, const int* seg_seq, const int* seg_pos0, const int* seg_rows, int n,
                           cudaStream_t stream);
int arcb_launch_feed(const StepState& st, const int* seqs, const int* tokens, int n, cudaStream_t stream);
// dst row = row_off + (r / rb) * rbp + r % rb, dst column = (c / cb) * cbp + c % cb, pitch dst_pitch;
// container 0 = bfloat16, 1 = half holding the bf16-rounded value, 2 = fp32
int arcb_launch_pack_blocks(const float* src, void* dst, long long rows, long long cols, int rb, int rbp, int row_off,
                            int cb, int cbp, long long dst_pitch, int container, cudaStream_t stream);
// the transpose of every head's block: element (h * rb + d, c) goes to row h * rbp + c, column d
int arcb_launch_pack_heads_t(const float* src, void* dst, int heads, int rb, int rbp, int cols, long long dst_pitch, int container,
                             cudaStream_t stream);
void arcb_count_launch(long long n);
