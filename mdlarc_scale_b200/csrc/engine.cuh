// Engine and session objects behind the C ABI, shared by engine.cu (the TinyTransformer path and the entry
// points) and layered.cu (models described as a list of layers).
#pragma once
#include <string>
#include <vector>

#include "../../include/arcb200.h"
#include "common.cuh"
#include "rowops.cuh"

int arcb_fail(int code, const char* msg);
int arcb_fail_cuda(cudaError_t e, const char* where);
#define CK(call)                                              \
  do {                                                        \
    cudaError_t e__ = (call);                                 \
    if (e__ != cudaSuccess) return arcb_fail_cuda(e__, #call); \
  } while (0)
#define CKL(expr, what)                                                          \
  do {                                                                           \
    int r__ = (expr);                                                            \
    if (r__ != 0) {                                                              \
      if (r__ > 0 && r__ < 1000) return arcb_fail_cuda((cudaError_t)r__, what);  \
      return arcb_fail(r__ < 0 ? ARCB_E_ARG : r__, what);                        \
    }                                                                            \
  } while (0)

struct LayeredModel;     // layered.cu
struct LayeredSession;

// GEMM weights hold the bf16-rounded parameter values in the 16-bit container of the activations
// (half or bfloat16), because the tensor-core MMA needs both operands in one format.
struct LayerWeights {
  float* ln1_w = nullptr;
  uint16_t* w_qkv = nullptr;   // [3d][d]
  uint16_t* w_out = nullptr;   // [d][d]
  float* ln2_w = nullptr;
  uint16_t* w_gu = nullptr;    // [2 dff][d], 64 gate rows then the matching 64 up rows, repeated
  float* b_gu = nullptr;       // [2 dff] packed the same way
  uint16_t* w_down = nullptr;  // [d][dff]
  float* b_down = nullptr;          // [d]
};

struct arcb_engine {
  arcb_config cfg;
  int device = 0;
  std::vector<LayerWeights> layers;
  float* token_embed = nullptr;
  float* example_embed = nullptr;
  float* lnf_w = nullptr;
  float* lm_head = nullptr;
  float* rope = nullptr;  // cos_x | sin_x | cos_y | sin_y | cos_z | sin_z
  int* d_err = nullptr;
  std::vector<void*> allocs;
  std::vector<char> loaded;  // [ARCB_T_COUNT * max(L,1)]
  LayeredModel* lm = nullptr;   // set: the network is a list of layers and everything above but d_err / allocs is unused
  bool act_f16() const { return cfg.act_format == ARCB_ACT_F16; }
};

struct arcb_session {
  arcb_engine* eng = nullptr;
  arcb_session_desc desc;
  int splits = 1;
  // workspace carve-up
  float* x = nullptr;
  uint16_t* xn16 = nullptr;
  uint16_t* q16 = nullptr;
  uint16_t* attn16 = nullptr;
  uint16_t* h16 = nullptr;
  uint16_t* k16 = nullptr;  // K/V of one prefill call in the activation format
  uint16_t* v16 = nullptr;
  float* attn_scratch = nullptr;
  float* gemm_scratch = nullptr;   // split-K partials of the decode step's residual GEMMs
  int* example_ids = nullptr;
  bool use_examples = false;
  DecodeState st{};
  cudaGraph_t graph = nullptr;
  cudaGraphExec_t graph_exec = nullptr;
  cudaStream_t capture_stream = nullptr;
  long long graph_kernels = 0;
  bool armed = false;
  // event pair recorded (as graph nodes) around the layer-0 decode-attention launch of every replay
  cudaEvent_t probe_begin = nullptr, probe_end = nullptr;
  bool probe_recorded = false;
  // the integer state block is cleared by the first arcb_prefill, on that call's stream
  int* state_ints = nullptr;
  size_t n_state_ints = 0;
  bool state_cleared = false;
  LayeredSession* ls = nullptr;   // set when the engine is layered
};

inline size_t align_up(size_t v, size_t a) { return (v + a - 1) / a * a; }

template <typename T>
inline int dev_alloc(arcb_engine* e, T** out, size_t count) {
  void* p = nullptr;
  cudaError_t r = cudaMalloc(&p, count * sizeof(T));
  if (r != cudaSuccess) return (int)r;
  e->allocs.push_back(p);
  *out = reinterpret_cast<T*>(p);
  return 0;
}


// layered.cu
void lm_destroy(LayeredModel* m);
int lm_load_tensor(arcb_engine* e, int kind, int layer, const float* src, long long numel, cudaStream_t stream);
bool lm_complete(const arcb_engine* e);
int64_t lm_cache_bytes(const arcb_engine* e, int n_seqs, int t_max);
int64_t lm_workspace_bytes(const arcb_engine* e, int n_seqs, int max_prefill_tokens, int attn_splits);
int lm_session_create(arcb_session* s);
void lm_session_destroy(LayeredSession* ls);
int lm_prefill(arcb_session* s, const arcb_prefill_args* a, cudaStream_t stream);
int lm_record_step(arcb_session* s, cudaStream_t stream);
int* lm_n_finished(arcb_session* s);
bool lm_armed(const arcb_session* s);
