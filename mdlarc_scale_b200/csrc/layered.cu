// Layered models: the network is data (a list of mixers and feed-forwards).  Weight packing, cache and
// state layout, workspace, and the forward pass shared by prefill and the captured decode step.
//
// Padding: the residual width, the feed-forward width and the vocabulary are rounded up to 128 columns
// and every head to 64, 128 or 256; padded weights, gains and biases are zero, so padded columns carry
// exact zeros and every product meets the tensor-core tile sizes whatever the model's sizes are.
#include <cstring>

#include "attn_gqa.cuh"
#include "attn_prefill_gqa.cuh"
#include "engine.cuh"
#include "gemm.cuh"
#include "layerops.cuh"
#include "mlstm.cuh"

namespace {

int pad128(int v) { return (v + 127) / 128 * 128; }
int pad_head(int d) { return d <= 64 ? 64 : d <= 128 ? 128 : 256; }

struct LmLayer {
  arcb_layer_desc d;
  int dimp, vdimp, ffp;
  bool own_kv;                 // attention with key/value projections of its own
  int off_q, off_k, off_v, off_g, off_gate, n_proj, k_out;
  float* norm1 = nullptr;
  float* norm2 = nullptr;
  void* w_proj = nullptr;      // [n_proj][Wp]
  float* b_proj = nullptr;     // [n_proj]
  float* q_norm = nullptr;
  float* k_norm = nullptr;
  float* sink = nullptr;
  float* head_norm = nullptr;  // [H * vdimp]
  void* w_out = nullptr;       // [Wp][H * vdimp]
  void* w_up = nullptr;        // [ffp][Wp]
  void* w_down = nullptr;      // [Wp][ffp]
};

}  // namespace

struct LayeredModel {
  arcb_model_desc d;
  int wp, vp, fmt, es;
  std::vector<LmLayer> layers;
  float* embed = nullptr;      // [vocab][Wp] fp32
  float* final_norm = nullptr;
  void* head = nullptr;        // [Vp][Wp]
  int n_proj_max = 0, heads_max = 0, k_out_max = 0, ffp_max = 0;
};

struct LayeredSession {
  float* x = nullptr;
  void* xn = nullptr;
  void* proj = nullptr;        // [R][n_proj] activation format: queries, recurrence k / v, sigmoid gates
  float* proj32 = nullptr;     // [R][n_proj] unfused projections
  float* gates = nullptr;      // [R][2 H]
  void* mix = nullptr;         // [R][H * vdimp]
  void* hid = nullptr;         // [R][ffp]
  void* hn = nullptr;          // [head_rows][Wp]
  float* logits = nullptr;     // [head_rows][Vp]
  float* attn_scratch = nullptr;
  float* gemm_scratch = nullptr;
  int head_rows = 0, splits = 1;
  int* ints = nullptr;
  size_t n_ints = 0;
  bool cleared = false, armed = false;
  StepState st{};
  std::vector<void*> k, v;     // per layer: keys and values (its own or the shared layer's)
  std::vector<float*> S, n, m; // per layer: recurrent state
};

namespace {

struct LmWs {
  size_t x, xn, proj, proj32, gates, mix, hid, hn, logits, ascratch, gscratch, ints, total;
  size_t n_ints;
  int head_rows;
};

// Head norms, gates and cache writes inside the projection product: the tensor-core kernels in a 16-bit
// format, heads that fit a column tile.
bool use_fused(const LayeredModel& m) {
  if (m.fmt == 2 || m.d.gemm_path == ARCB_GEMM_SIMT || !m.d.fused_proj) return false;
  for (const LmLayer& L : m.layers)
    if (L.d.mixer == ARCB_MIXER_ATTENTION && L.d.qk_norm && L.dimp > 128) return false;
  return true;
}

int lm_splits(const LayeredModel& m, int B, int requested, int t_max) {
  if (requested > 0) return requested > 64 ? 64 : requested;
  int s = 1;
  for (const LmLayer& L : m.layers)
    if (L.d.mixer == ARCB_MIXER_ATTENTION) {
      const int c = arcb_attn_gqa_splits(B, L.d.kv_heads, L.d.heads / L.d.kv_heads, t_max);
      s = c > s ? c : s;
    }
  return s;
}

LmWs lm_ws(const LayeredModel& m, int B, int P, int splits) {
  const size_t R = (size_t)(B > P ? B : P);
  LmWs w;
  w.head_rows = B > 1024 ? B : (P < 1024 ? (P > B ? P : B) : 1024);
  size_t off = 0;
  auto take = [&](size_t bytes) { const size_t at = off; off = align_up(off + bytes, 1024); return at; };
  w.x = take(R * m.wp * 4);
  w.xn = take(R * m.wp * m.es);
  w.proj = take(R * m.n_proj_max * m.es);
  w.proj32 = take(use_fused(m) ? 0 : R * m.n_proj_max * 4);
  w.gates = take(R * 2 * m.heads_max * 4);
  w.mix = take(R * m.k_out_max * m.es);
  w.hid = take(R * (size_t)m.ffp_max * m.es);
  w.hn = take((size_t)w.head_rows * m.wp * m.es);
  w.logits = take((size_t)w.head_rows * m.vp * 4);
  w.ascratch = take(splits > 1 ? (size_t)B * m.heads_max * splits * (256 + 4) * 4 : 0);
  w.gscratch = take(align_up((size_t)B, 128) * m.wp * 4);
  w.n_ints = (size_t)B * 7 + 64;
  w.ints = take(w.n_ints * 4);
  w.total = off;
  return w;
}

size_t kv_plane(const LayeredModel& m, const LmLayer& L, int B, int T, bool value) {
  return align_up((size_t)B * L.d.kv_heads * T * (value ? L.vdimp : L.dimp) * m.es, 1024);
}
size_t st_plane(const LmLayer& L, int B, int which) {   // 0 S, 1 n, 2 m
  const size_t per = which == 0 ? (size_t)L.d.dim * L.vdimp : which == 1 ? L.dimp : 1;
  return align_up((size_t)B * L.d.heads * per * 4, 1024);
}

// dev_alloc of zeroed memory (padding must be zero)
template <typename T>
int zalloc(arcb_engine* e, T** out, size_t bytes) {
  uint8_t* p = nullptr;
  const int r = dev_alloc(e, &p, bytes);
  if (r) return r;
  *out = reinterpret_cast<T*>(p);
  return (int)cudaMemset(p, 0, bytes);
}

}  // namespace

extern "C" int arcb_engine_create_layered(const arcb_model_desc* md, const arcb_layer_desc* ld, arcb_engine** out) {
  if (!md || !ld || !out) return arcb_fail(ARCB_E_ARG, "null argument");
  if (md->width <= 0 || md->vocab <= 0 || md->n_layers <= 0) return arcb_fail(ARCB_E_ARG, "bad model sizes");
  if (md->act_format < ARCB_ACT_F16 || md->act_format > ARCB_ACT_F32) return arcb_fail(ARCB_E_ARG, "unknown act_format");
  if (md->norm != ARCB_NORM_LAYER && md->norm != ARCB_NORM_RMS) return arcb_fail(ARCB_E_UNSUPPORTED, "unknown norm");
  for (int l = 0; l < md->n_layers; ++l) {
    const arcb_layer_desc& d = ld[l];
    if (d.heads <= 0 || d.dim <= 0 || d.vdim <= 0) return arcb_fail(ARCB_E_ARG, "bad head sizes");
    if (d.dim > 256 || d.vdim > 256) return arcb_fail(ARCB_E_UNSUPPORTED, "head sizes above 256 are not implemented");
    if (d.mixer == ARCB_MIXER_ATTENTION) {
      if (d.kv_heads <= 0 || d.heads % d.kv_heads) return arcb_fail(ARCB_E_ARG, "kv_heads must divide heads");
      if (d.q_temp_every < 0) return arcb_fail(ARCB_E_ARG, "q_temp_every must not be negative");
      if (d.kv_from >= 0) {
        if (d.kv_from >= l) return arcb_fail(ARCB_E_ARG, "kv_from must name an earlier layer");
        const arcb_layer_desc& s = ld[d.kv_from];
        if (s.mixer != ARCB_MIXER_ATTENTION || s.kv_from >= 0 || s.kv_heads != d.kv_heads || s.dim != d.dim || s.vdim != d.vdim)
          return arcb_fail(ARCB_E_ARG, "kv_from must name an attention layer with its own keys and the same head sizes");
      }
    } else if (d.mixer == ARCB_MIXER_MLSTM) {
      if (!(d.gate_cap > 0.f)) return arcb_fail(ARCB_E_ARG, "gate_cap must be positive");
    } else {
      return arcb_fail(ARCB_E_UNSUPPORTED, "unknown mixer");
    }
    if (d.mlp != ARCB_MLP_NONE && (d.mlp != ARCB_MLP_RELU2 || d.d_ff <= 0))
      return arcb_fail(ARCB_E_UNSUPPORTED, "unknown feed-forward");
  }
  if (!arcb_device_ok()) return arcb_fail(ARCB_E_UNSUPPORTED, "current device is not compute capability 10.x");
  CKL(arcb_gemm_init(), "gemm init (shared-memory opt-in / cuTensorMapEncodeTiled lookup)");
  CKL(arcb_mlstm_chunk_init(), "chunkwise recurrence init (shared-memory opt-in)");
  CKL(arcb_attn_prefill_gqa_init(), "prefill attention init (shared-memory opt-in)");
  arcb_engine* e = new arcb_engine();
  std::memset(&e->cfg, 0, sizeof e->cfg);
  cudaGetDevice(&e->device);
  LayeredModel* m = new LayeredModel();
  e->lm = m;
  m->d = *md;
  m->wp = pad128(md->width);
  m->vp = pad128(md->vocab);
  m->fmt = md->act_format == ARCB_ACT_F32 ? 2 : md->act_format == ARCB_ACT_F16 ? 1 : 0;
  m->es = act_bytes(m->fmt);
  e->loaded.assign((size_t)ARCB_L_COUNT * md->n_layers, 0);
  int r = 0;
  for (int l = 0; l < md->n_layers; ++l) {
    LmLayer L;
    L.d = ld[l];
    const arcb_layer_desc& d = L.d;
    const bool rec = d.mixer == ARCB_MIXER_MLSTM;
    L.dimp = pad_head(d.dim);
    L.vdimp = pad_head(d.vdim);
    L.ffp = d.mlp == ARCB_MLP_NONE ? 0 : pad128(d.d_ff);
    L.own_kv = !rec && d.kv_from < 0;
    L.k_out = d.heads * L.vdimp;
    const int nkv = rec ? d.heads : d.kv_heads;
    int at = 0;
    L.off_q = at; at += d.heads * L.dimp;
    L.off_k = L.off_v = L.off_g = L.off_gate = -1;
    if (rec || L.own_kv) {
      L.off_k = at; at += nkv * L.dimp;
      L.off_v = at; at += nkv * L.vdimp;
    }
    if (rec || d.out_gate) { L.off_g = at; at += d.heads * L.vdimp; }
    if (rec) { L.off_gate = at; at += 2 * d.heads; }
    L.n_proj = pad128(at);
    r |= zalloc(e, &L.norm1, (size_t)m->wp * 4);
    r |= zalloc(e, &L.w_proj, (size_t)L.n_proj * m->wp * m->es);
    r |= zalloc(e, &L.b_proj, (size_t)L.n_proj * 4);
    r |= zalloc(e, &L.q_norm, (size_t)L.dimp * 4);
    r |= zalloc(e, &L.k_norm, (size_t)L.dimp * 4);
    r |= zalloc(e, &L.sink, (size_t)d.heads * 4);
    r |= zalloc(e, &L.head_norm, (size_t)L.k_out * 4);
    r |= zalloc(e, &L.w_out, (size_t)m->wp * L.k_out * m->es);
    if (L.ffp) {
      r |= zalloc(e, &L.norm2, (size_t)m->wp * 4);
      r |= zalloc(e, &L.w_up, (size_t)L.ffp * m->wp * m->es);
      r |= zalloc(e, &L.w_down, (size_t)m->wp * L.ffp * m->es);
    }
    m->n_proj_max = L.n_proj > m->n_proj_max ? L.n_proj : m->n_proj_max;
    m->heads_max = d.heads > m->heads_max ? d.heads : m->heads_max;
    m->k_out_max = L.k_out > m->k_out_max ? L.k_out : m->k_out_max;
    m->ffp_max = L.ffp > m->ffp_max ? L.ffp : m->ffp_max;
    m->layers.push_back(L);
  }
  r |= zalloc(e, &m->embed, (size_t)md->vocab * m->wp * 4);
  r |= zalloc(e, &m->final_norm, (size_t)m->wp * 4);
  r |= zalloc(e, &m->head, (size_t)m->vp * m->wp * m->es);
  r |= dev_alloc(e, &e->d_err, 64);
  if (!r) r = (int)cudaMemset(e->d_err, 0, 64 * sizeof(int));
  if (!r) r = (int)cudaDeviceSynchronize();   // the zero fills precede the loads, which use other streams
  if (r) {
    arcb_engine_destroy(e);
    return arcb_fail(ARCB_E_STATE, "cudaMalloc of packed weights failed");
  }
  *out = e;
  return ARCB_OK;
}

void lm_destroy(LayeredModel* m) { delete m; }

int lm_load_tensor(arcb_engine* e, int kind, int layer, const float* src, long long numel, cudaStream_t stream) {
  LayeredModel& m = *e->lm;
  if (kind < 0 || kind >= ARCB_L_COUNT) return arcb_fail(ARCB_E_ARG, "unknown tensor kind");
  const bool per_layer = kind >= ARCB_L_NORM1;
  if (per_layer && (layer < 0 || layer >= m.d.n_layers)) return arcb_fail(ARCB_E_ARG, "layer out of range");
  LmLayer* L = per_layer ? &m.layers[layer] : nullptr;
  const long long W = m.d.width;
  // destination: rows in blocks rb -> rbp from row_off, columns in blocks cb -> cbp, `pitch` columns
  long long rows = 0, cols = 0, pitch = 0;
  int rb = 0, rbp = 0, row_off = 0, cb = 0, cbp = 0;
  void* dst = nullptr;
  bool weight = true;          // matrices in the operand format, everything else fp32
  const bool rec = L && L->d.mixer == ARCB_MIXER_MLSTM;
  const int H = L ? L->d.heads : 0, nkv = L ? (rec ? H : L->d.kv_heads) : 0;
  auto rows_of = [&](int heads, int size, int padded, int off) {
    rows = (long long)heads * size; rb = size; rbp = padded; row_off = off; cols = W; pitch = m.wp; dst = L->w_proj;
  };
  auto bias_of = [&](int heads, int size, int padded, int off) {
    rows_of(heads, size, padded, off);
    cols = 1; pitch = 1; dst = L->b_proj; weight = false;
  };
  auto vec = [&](float* p, long long n) { rows = 1; cols = n; pitch = n; dst = p; weight = false; };
  switch (kind) {
    case ARCB_L_EMBED: rows = m.d.vocab; cols = W; pitch = m.wp; dst = m.embed; weight = false; break;
    case ARCB_L_FINAL_NORM: vec(m.final_norm, W); break;
    case ARCB_L_HEAD: rows = m.d.vocab; cols = W; pitch = m.wp; dst = m.head; break;
    case ARCB_L_NORM1: vec(L->norm1, W); break;
    case ARCB_L_NORM2: if (L->ffp) vec(L->norm2, W); break;
    case ARCB_L_Q: rows_of(H, L->d.dim, L->dimp, L->off_q); break;
    case ARCB_L_Q_B: bias_of(H, L->d.dim, L->dimp, L->off_q); break;
    case ARCB_L_K: if (L->off_k >= 0) rows_of(nkv, L->d.dim, L->dimp, L->off_k); break;
    case ARCB_L_K_B: if (L->off_k >= 0) bias_of(nkv, L->d.dim, L->dimp, L->off_k); break;
    case ARCB_L_V: if (L->off_v >= 0) rows_of(nkv, L->d.vdim, L->vdimp, L->off_v); break;
    case ARCB_L_V_B: if (L->off_v >= 0) bias_of(nkv, L->d.vdim, L->vdimp, L->off_v); break;
    case ARCB_L_G: if (L->off_g >= 0) rows_of(H, L->d.vdim, L->vdimp, L->off_g); break;
    case ARCB_L_O: rows = W; cols = (long long)H * L->d.vdim; cb = L->d.vdim; cbp = L->vdimp; pitch = L->k_out; dst = L->w_out; break;
    case ARCB_L_Q_NORM: vec(L->q_norm, L->d.dim); break;
    case ARCB_L_K_NORM: vec(L->k_norm, L->d.dim); break;
    case ARCB_L_SINK: vec(L->sink, H); break;
    case ARCB_L_HEAD_NORM: vec(L->head_norm, (long long)H * L->d.vdim); cb = L->d.vdim; cbp = L->vdimp; break;
    case ARCB_L_I: if (rec) rows_of(1, H, H, L->off_gate); break;
    case ARCB_L_I_B: if (rec) bias_of(1, H, H, L->off_gate); break;
    case ARCB_L_F: if (rec) rows_of(1, H, H, L->off_gate + H); break;
    case ARCB_L_F_B: if (rec) bias_of(1, H, H, L->off_gate + H); break;
    case ARCB_L_UP: if (L->ffp) { rows = L->d.d_ff; cols = W; pitch = m.wp; dst = L->w_up; } break;
    case ARCB_L_DOWN: if (L->ffp) { rows = W; cols = L->d.d_ff; pitch = L->ffp; dst = L->w_down; } break;
  }
  if (!dst) return arcb_fail(ARCB_E_ARG, "this layer has no such tensor");
  if (numel != rows * cols) return arcb_fail(ARCB_E_ARG, "tensor has the wrong number of elements");
  if (!rb) { rb = (int)rows; rbp = rb; }
  if (!cb) { cb = (int)cols; cbp = cb; }
  CKL(arcb_launch_pack_blocks(src, dst, rows, cols, rb, rbp, row_off, cb, cbp, pitch, weight ? m.fmt : 2, stream), "pack_blocks");
  e->loaded[(size_t)kind * m.d.n_layers + (per_layer ? layer : 0)] = 1;
  return ARCB_OK;
}

bool lm_complete(const arcb_engine* e) {
  const LayeredModel& m = *e->lm;
  auto has = [&](int kind, int l) { return e->loaded[(size_t)kind * m.d.n_layers + l] != 0; };
  if (!has(ARCB_L_EMBED, 0) || !has(ARCB_L_FINAL_NORM, 0) || !has(ARCB_L_HEAD, 0)) return false;
  for (int l = 0; l < m.d.n_layers; ++l) {
    const LmLayer& L = m.layers[l];
    const bool rec = L.d.mixer == ARCB_MIXER_MLSTM;
    bool ok = has(ARCB_L_NORM1, l) && has(ARCB_L_Q, l) && has(ARCB_L_O, l);
    if (rec || L.own_kv) ok = ok && has(ARCB_L_K, l) && has(ARCB_L_V, l);
    if (L.off_g >= 0) ok = ok && has(ARCB_L_G, l);
    if (rec) ok = ok && has(ARCB_L_I, l) && has(ARCB_L_I_B, l) && has(ARCB_L_F, l) && has(ARCB_L_F_B, l) && has(ARCB_L_HEAD_NORM, l);
    if (L.d.qkv_bias) ok = ok && has(ARCB_L_Q_B, l) && (!L.own_kv || (has(ARCB_L_K_B, l) && has(ARCB_L_V_B, l)));
    if (!rec && L.d.qk_norm) ok = ok && has(ARCB_L_Q_NORM, l) && (!L.own_kv || has(ARCB_L_K_NORM, l));
    if (!rec && L.d.sink) ok = ok && has(ARCB_L_SINK, l);
    if (L.ffp) ok = ok && has(ARCB_L_NORM2, l) && has(ARCB_L_UP, l) && has(ARCB_L_DOWN, l);
    if (!ok) return false;
  }
  return true;
}

// ---------------------------------------------------------------------------
// session
// ---------------------------------------------------------------------------
int64_t lm_cache_bytes(const arcb_engine* e, int B, int T) {
  const LayeredModel& m = *e->lm;
  size_t n = 0;
  for (const LmLayer& L : m.layers) {
    if (L.own_kv) n += kv_plane(m, L, B, T, false) + kv_plane(m, L, B, T, true);
    if (L.d.mixer == ARCB_MIXER_MLSTM) n += st_plane(L, B, 0) + st_plane(L, B, 1) + st_plane(L, B, 2);
  }
  return (int64_t)(n ? n : 1024);
}

int64_t lm_workspace_bytes(const arcb_engine* e, int B, int P, int attn_splits) {
  return (int64_t)lm_ws(*e->lm, B, P, lm_splits(*e->lm, B, attn_splits, 0)).total;
}

int lm_session_create(arcb_session* s) {
  const LayeredModel& m = *s->eng->lm;
  const arcb_session_desc& d = s->desc;
  const int B = d.n_seqs, T = d.t_max;
  LayeredSession* ls = new LayeredSession();
  s->ls = ls;
  ls->splits = lm_splits(m, B, d.attn_splits, T);
  const LmWs w = lm_ws(m, B, d.max_prefill_tokens, lm_splits(m, B, d.attn_splits, 0));
  uint8_t* base = reinterpret_cast<uint8_t*>(d.d_workspace);
  ls->x = reinterpret_cast<float*>(base + w.x);
  ls->xn = base + w.xn;
  ls->proj = base + w.proj;
  ls->proj32 = reinterpret_cast<float*>(base + w.proj32);
  ls->gates = reinterpret_cast<float*>(base + w.gates);
  ls->mix = base + w.mix;
  ls->hid = base + w.hid;
  ls->hn = base + w.hn;
  ls->logits = reinterpret_cast<float*>(base + w.logits);
  ls->attn_scratch = ls->splits > 1 ? reinterpret_cast<float*>(base + w.ascratch) : nullptr;
  ls->gemm_scratch = reinterpret_cast<float*>(base + w.gscratch);
  ls->head_rows = w.head_rows;
  ls->ints = reinterpret_cast<int*>(base + w.ints);
  ls->n_ints = w.n_ints;
  StepState& st = ls->st;
  st.n_seqs = B; st.t_max = T; st.max_new = d.max_new; st.stop_on_end = d.stop_on_end; st.end_token = d.end_token;
  int* p = ls->ints;
  st.cur_len = p; st.len0 = p + B; st.cur_tok = p + 2 * B; st.active = p + 3 * B; st.pos = p + 4 * B;
  st.kv_len = p + 5 * B; st.finished = p + 6 * B; st.n_finished = p + 7 * B;
  st.out_tokens = d.d_out_tokens; st.forced = d.d_forced; st.step_logits = d.d_step_logits;
  st.temperature = d.temperature; st.top_k = d.top_k; st.sample_seed = d.sample_seed; st.sample_stream = d.d_sample_stream;
  st.err = s->eng->d_err;
  uint8_t* c = reinterpret_cast<uint8_t*>(d.d_kv_cache);
  const size_t L = m.layers.size();
  ls->k.assign(L, nullptr); ls->v.assign(L, nullptr);
  ls->S.assign(L, nullptr); ls->n.assign(L, nullptr); ls->m.assign(L, nullptr);
  for (size_t l = 0; l < L; ++l) {
    const LmLayer& y = m.layers[l];
    if (y.own_kv) {
      ls->k[l] = c; c += kv_plane(m, y, B, T, false);
      ls->v[l] = c; c += kv_plane(m, y, B, T, true);
    } else if (y.d.mixer == ARCB_MIXER_ATTENTION) {
      ls->k[l] = ls->k[y.d.kv_from];
      ls->v[l] = ls->v[y.d.kv_from];
    } else {
      ls->S[l] = reinterpret_cast<float*>(c); c += st_plane(y, B, 0);
      ls->n[l] = reinterpret_cast<float*>(c); c += st_plane(y, B, 1);
      ls->m[l] = reinterpret_cast<float*>(c); c += st_plane(y, B, 2);
    }
  }
  return ARCB_OK;
}

void lm_session_destroy(LayeredSession* ls) { delete ls; }
int* lm_n_finished(arcb_session* s) { return s->ls->st.n_finished; }
bool lm_armed(const arcb_session* s) { return s->ls->armed; }

// ---------------------------------------------------------------------------
// forward pass
// ---------------------------------------------------------------------------
namespace {

bool lm_tc(const LayeredModel& m) { return m.fmt != 2 && m.d.gemm_path != ARCB_GEMM_SIMT; }

int lm_gemm(const LayeredModel& m, const void* a, const void* w, GemmEpilogue& ep, int K, cudaStream_t stream) {
  return arcb_launch_gemm(a, w, ep, K, m.fmt, lm_tc(m), stream);
}

// Rows of one pass through the layers: a prefill call's packed tokens, or one row per sequence of a step.
struct Rows {
  int n;
  const int* pos;              // position of each row, < 0: held
  const int* seq;              // cache row, null: row index
  const int* kv_len;           // visible keys
  const arcb_prefill_args* pa; // null in a decode step
};

int lm_residual(arcb_session* s, const void* a, const void* w, int K, int rows, bool step, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  GemmEpilogue er{};
  er.mode = EPI_RESID; er.M = rows; er.N = m.wp; er.x = s->ls->x; er.act_f16 = m.fmt; er.err = s->eng->d_err;
  er.splitk_scratch = step ? s->ls->gemm_scratch : nullptr;
  CKL(lm_gemm(m, a, w, er, K, stream), "residual gemm");
  return ARCB_OK;
}

int lm_norm(arcb_session* s, const float* w, int rows, float x_scale, float* dense, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  LmNormArgs a{};
  a.kind = m.d.norm; a.rows = rows; a.width = m.d.width; a.pitch = m.wp; a.fmt = m.fmt; a.eps = m.d.norm_eps;
  a.x_scale = x_scale; a.x = s->ls->x; a.w = w; a.xn = s->ls->xn; a.write_x = 1; a.dense = dense;
  CKL(arcb_launch_lm_norm(a, stream), "norm");
  return ARCB_OK;
}

int lm_mixer(arcb_session* s, int l, const Rows& R, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  LayeredSession* ls = s->ls;
  const LmLayer& L = m.layers[l];
  const arcb_layer_desc& d = L.d;
  const bool rec = d.mixer == ARCB_MIXER_MLSTM;
  const int B = s->desc.n_seqs, T = s->desc.t_max;

  ProjArgs p{};
  p.recurrent = rec ? 1 : 0; p.M = R.n; p.N = L.n_proj; p.H = d.heads; p.G = rec ? d.heads : d.kv_heads;
  p.dim = d.dim; p.dimp = L.dimp; p.vdim = d.vdim; p.vdimp = L.vdimp;
  p.off_q = L.off_q; p.off_k = L.off_k; p.off_v = L.off_v; p.off_g = L.off_g; p.off_gate = L.off_gate;
  p.bias = (d.qkv_bias || rec) ? L.b_proj : nullptr;
  p.q_norm = (!rec && d.qk_norm) ? L.q_norm : nullptr;
  p.k_norm = (!rec && d.qk_norm) ? L.k_norm : nullptr;
  p.eps = m.d.norm_eps;
  p.q_mul = rec ? 1.f / sqrtf((float)d.dim) : 1.f;
  p.temp_coef = d.q_temp_coef; p.temp_every = rec ? 0 : d.q_temp_every;
  p.pos = R.pos; p.seq = R.seq; p.kcache = ls->k[l]; p.vcache = ls->v[l]; p.t_max = T; p.n_seqs = B;
  p.out = ls->proj; p.gates = ls->gates; p.fmt = m.fmt; p.err = s->eng->d_err;
  GemmEpilogue ep{};
  ep.M = R.n; ep.N = L.n_proj; ep.act_f16 = m.fmt; ep.err = s->eng->d_err;
  if (use_fused(m)) {
    ep.mode = EPI_HEADS; ep.pj = p;
    CKL(lm_gemm(m, ls->xn, L.w_proj, ep, m.wp, stream), "fused projection gemm");
  } else {
    ep.mode = EPI_STORE_F32; ep.y = ls->proj32;
    CKL(lm_gemm(m, ls->xn, L.w_proj, ep, m.wp, stream), "projection gemm");
    CKL(arcb_launch_proj_prep(p, ls->proj32, stream), "projection prep");
  }

  if (rec) {
    MlstmArgs a{};
    a.proj = ls->proj; a.pitch = L.n_proj; a.off_q = L.off_q; a.off_k = L.off_k; a.off_v = L.off_v; a.off_g = L.off_g;
    a.gates = ls->gates; a.gate_cap = d.gate_cap; a.norm_w = L.head_norm; a.out = ls->mix; a.S = ls->S[l]; a.n = ls->n[l]; a.m = ls->m[l];
    a.H = d.heads; a.dim = d.dim; a.dimp = L.dimp; a.vdim = d.vdim; a.vdimp = L.vdimp; a.n_seqs = B; a.fmt = m.fmt;
    a.n_rows = R.n; a.eps = m.d.norm_eps; a.err = s->eng->d_err;
    if (R.pa) {
      a.seg_row0 = R.pa->d_seg_row0; a.seg_rows = R.pa->d_seg_rows; a.seg_seq = R.pa->d_seg_seq; a.seg_pos0 = R.pa->d_seg_pos0;
      a.n_segs = R.pa->n_segs;
    } else {
      a.pos = R.pos; a.n_segs = R.n;
    }
    if (R.pa && m.d.mlstm_path == ARCB_MLSTM_AUTO && arcb_mlstm_chunk_supported(L.dimp, L.vdimp, m.fmt))
      CKL(arcb_launch_mlstm_chunk(a, stream), "mlstm chunks");
    else
      CKL(arcb_launch_mlstm_step(a, stream), "mlstm");
  } else if (R.pa && m.fmt != 2 && m.d.attn_path == ARCB_ATTN_AUTO && R.pa->n_qblocks > 0 &&
             arcb_attn_prefill_gqa_supported(L.dimp, L.vdimp, B, d.kv_heads, T, d.scale)) {
    AttnPrefillGqaArgs a{};
    a.q = ls->proj; a.q_pitch = L.n_proj; a.q_col = L.off_q; a.k = ls->k[l]; a.v = ls->v[l];
    if (L.off_g >= 0) { a.gate = reinterpret_cast<const uint8_t*>(ls->proj) + (size_t)L.off_g * m.es; a.gate_pitch = L.n_proj; }
    a.out = ls->mix; a.seq = R.seq; a.kv_count = R.kv_len; a.qblock_row0 = R.pa->d_qblock_row0; a.qblock_rows = R.pa->d_qblock_rows;
    a.sink = d.sink ? L.sink : nullptr; a.n_qblocks = R.pa->n_qblocks; a.n_rows = R.n; a.n_heads = d.heads; a.n_kv = d.kv_heads;
    a.dimp = L.dimp; a.vdimp = L.vdimp; a.t_max = T; a.n_seqs = B; a.scale = d.scale; a.act_f16 = m.fmt; a.err = s->eng->d_err;
    CKL(arcb_launch_attn_prefill_gqa(a, stream), "prefill attention");
  } else {
    AttnGqaArgs a{};
    const uint8_t* pr = reinterpret_cast<const uint8_t*>(ls->proj);
    a.q = pr + (size_t)L.off_q * m.es; a.q_pitch = L.n_proj; a.k = ls->k[l]; a.v = ls->v[l];
    if (L.off_g >= 0) { a.gate = pr + (size_t)L.off_g * m.es; a.gate_pitch = L.n_proj; }
    a.out = ls->mix; a.item_seq = R.seq; a.item_len = R.kv_len; a.sink = d.sink ? L.sink : nullptr;
    a.n_items = R.n; a.n_heads = d.heads; a.n_kv = d.kv_heads; a.dimp = L.dimp; a.vdimp = L.vdimp; a.t_max = T; a.n_seqs = B;
    a.n_splits = R.pa ? 1 : ls->splits; a.scale = d.scale; a.scratch = ls->attn_scratch; a.fmt = m.fmt; a.err = s->eng->d_err;
    CKL(arcb_launch_attn_gqa(a, stream), "attention");
  }
  return lm_residual(s, ls->mix, L.w_out, L.k_out, R.n, R.pa == nullptr, stream);
}

int lm_layers(arcb_session* s, const Rows& R, float* residuals, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  LayeredSession* ls = s->ls;
  for (int l = 0; l < m.d.n_layers; ++l) {
    const LmLayer& L = m.layers[l];
    const bool last = l + 1 == m.d.n_layers;
    float* dense = residuals ? residuals + (size_t)l * R.n * m.d.width : nullptr;
    int r = lm_mixer(s, l, R, stream);
    if (r) return r;
    // the norm leaves x already multiplied by the factor of the next sublayer's sum
    r = lm_norm(s, L.norm1, R.n, last && !L.ffp ? 1.f : m.d.residual_alpha, L.ffp ? nullptr : dense, stream);
    if (r) return r;
    if (L.ffp) {
      GemmEpilogue eu{};
      eu.mode = EPI_RELU2; eu.M = R.n; eu.N = L.ffp; eu.out16 = ls->hid; eu.act_f16 = m.fmt; eu.err = s->eng->d_err;
      CKL(lm_gemm(m, ls->xn, L.w_up, eu, m.wp, stream), "up gemm");
      r = lm_residual(s, ls->hid, L.w_down, L.ffp, R.n, R.pa == nullptr, stream);
      if (!r) r = lm_norm(s, L.norm2, R.n, last ? 1.f : m.d.residual_alpha, dense, stream);
      if (r) return r;
    }
  }
  return ARCB_OK;
}

// final norm and logits of `rows` rows of x (gathered by `index`) into ls->logits, then token picking
int lm_head(arcb_session* s, int mode, int rows, const int* index, float* out, const int* first_seq, const int* prompt_len,
            cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  LayeredSession* ls = s->ls;
  for (int r0 = 0; r0 < rows; r0 += ls->head_rows) {
    const int n = rows - r0 < ls->head_rows ? rows - r0 : ls->head_rows;
    LmNormArgs a{};
    a.kind = m.d.norm; a.rows = n; a.width = m.d.width; a.pitch = m.wp; a.fmt = m.fmt; a.eps = m.d.norm_eps;
    a.x_scale = 1.f; a.x = ls->x; a.w = m.final_norm; a.xn = ls->hn; a.write_x = 0; a.row_index = index ? index + r0 : nullptr;
    CKL(arcb_launch_lm_norm(a, stream), "final norm");
    GemmEpilogue ep{};
    ep.mode = EPI_STORE_F32; ep.M = n; ep.N = m.vp; ep.y = ls->logits; ep.act_f16 = m.fmt; ep.err = s->eng->d_err;
    CKL(lm_gemm(m, ls->hn, m.head, ep, m.wp, stream), "head gemm");
    PickArgs p{};
    p.mode = mode; p.rows = n; p.vocab = m.d.vocab; p.pitch = m.vp; p.logits = ls->logits; p.scale = m.d.logit_scale;
    p.out = out ? out + (size_t)r0 * m.d.vocab : nullptr;
    p.first_seq = first_seq ? first_seq + r0 : nullptr;
    p.prompt_len = prompt_len ? prompt_len + r0 : nullptr;
    CKL(arcb_launch_pick(p, ls->st, stream), "pick");
  }
  return ARCB_OK;
}

LmEmbedArgs lm_embed_args(const arcb_session* s, int rows, const int* tokens) {
  const LayeredModel& m = *s->eng->lm;
  LmEmbedArgs a{};
  a.rows = rows; a.width = m.d.width; a.pitch = m.wp; a.vocab = m.d.vocab; a.fmt = m.fmt; a.token_ids = tokens;
  a.embed = m.embed; a.alpha = m.d.residual_alpha; a.x = s->ls->x; a.xn = s->ls->xn;
  return a;
}

// The integer state, and the cache: rows a query does not see are still operands of a product whose
// weights are zero, so they must hold finite numbers.
int lm_clear(arcb_session* s, cudaStream_t stream) {
  LayeredSession* ls = s->ls;
  if (ls->cleared) return ARCB_OK;
  CK(cudaMemsetAsync(ls->ints, 0, ls->n_ints * 4, stream));
  CK(cudaMemsetAsync(s->desc.d_kv_cache, 0, (size_t)lm_cache_bytes(s->eng, s->desc.n_seqs, s->desc.t_max), stream));
  ls->cleared = true;
  return ARCB_OK;
}

}  // namespace

int lm_prefill(arcb_session* s, const arcb_prefill_args* a, cudaStream_t stream) {
  LayeredSession* ls = s->ls;
  if (!a->d_token_ids || !a->d_seq || !a->d_kv_slot || !a->d_kv_count) return arcb_fail(ARCB_E_ARG, "null token arrays");
  if (a->n_segs <= 0 || !a->d_seg_row0 || !a->d_seg_rows || !a->d_seg_seq || !a->d_seg_pos0)
    return arcb_fail(ARCB_E_ARG, "a layered prefill needs its segment list");
  if (a->n_first < 0 || (a->n_first > 0 && (!a->d_first_row || !a->d_first_seq || !a->d_prompt_len)))
    return arcb_fail(ARCB_E_ARG, "null first-token arrays");
  if (a->n_logit_rows < 0 || (a->n_logit_rows > 0 && (!a->d_logit_row || !a->d_logits)))
    return arcb_fail(ARCB_E_ARG, "null logit arrays");
  if (a->n_qblocks > 0 && (!a->d_qblock_row0 || !a->d_qblock_rows)) return arcb_fail(ARCB_E_ARG, "null query blocks");
  int r = lm_clear(s, stream);
  if (r) return r;
  CKL(arcb_launch_lm_embed(lm_embed_args(s, a->n_tokens, a->d_token_ids), stream), "embed");
  const Rows R{a->n_tokens, a->d_kv_slot, a->d_seq, a->d_kv_count, a};
  r = lm_layers(s, R, a->d_residuals, stream);
  if (r) return r;
  CKL(arcb_launch_seg_commit(ls->st, a->d_seg_seq, a->d_seg_pos0, a->d_seg_rows, a->n_segs, stream), "commit");
  if (a->d_logits_all) {
    r = lm_head(s, PICK_PLAIN, a->n_tokens, nullptr, a->d_logits_all, nullptr, nullptr, stream);
    if (r) return r;
  }
  if (a->n_logit_rows > 0) {
    r = lm_head(s, PICK_PLAIN, a->n_logit_rows, a->d_logit_row, a->d_logits, nullptr, nullptr, stream);
    if (r) return r;
  }
  if (a->n_first > 0) {
    r = lm_head(s, PICK_FIRST, a->n_first, a->d_first_row, a->d_first_logits, a->d_first_seq, a->d_prompt_len, stream);
    if (r) return r;
  }
  ls->armed = true;
  return ARCB_OK;
}

int lm_record_step(arcb_session* s, cudaStream_t stream) {
  LayeredSession* ls = s->ls;
  const int B = s->desc.n_seqs;
  CKL(arcb_launch_step_begin(ls->st, lm_embed_args(s, B, nullptr), stream), "step_begin");
  const Rows R{B, ls->st.pos, nullptr, ls->st.kv_len, nullptr};
  int r = lm_layers(s, R, nullptr, stream);
  if (r) return r;
  return lm_head(s, PICK_DECODE, B, nullptr, nullptr, nullptr, nullptr, stream);
}

extern "C" int arcb_session_feed(arcb_session* s, int32_t n, const int32_t* d_seqs, const int32_t* d_tokens, void* stream_v) {
  if (!s || !s->ls) return arcb_fail(ARCB_E_STATE, "arcb_session_feed needs a layered session");
  if (n <= 0 || !d_seqs || !d_tokens) return arcb_fail(ARCB_E_ARG, "nothing to feed");
  if (!s->ls->armed) return arcb_fail(ARCB_E_STATE, "arcb_prefill must run before arcb_session_feed");
  CKL(arcb_launch_feed(s->ls->st, d_seqs, d_tokens, n, (cudaStream_t)stream_v), "feed");
  return ARCB_OK;
}

extern "C" int arcb_session_step_logits(arcb_session* s, float** d_logits, int32_t* pitch) {
  if (!s || !s->ls || !d_logits || !pitch) return arcb_fail(ARCB_E_ARG, "arcb_session_step_logits needs a layered session");
  *d_logits = s->ls->logits;
  *pitch = s->eng->lm->vp;
  return ARCB_OK;
}

extern "C" int arcb_session_finished(arcb_session* s, int32_t* h_finished, void* stream_v) {
  if (!s || !s->ls || !h_finished) return arcb_fail(ARCB_E_ARG, "arcb_session_finished needs a layered session");
  cudaStream_t stream = (cudaStream_t)stream_v;
  CK(cudaMemcpyAsync(h_finished, s->ls->st.finished, (size_t)s->desc.n_seqs * 4, cudaMemcpyDeviceToHost, stream));
  CK(cudaStreamSynchronize(stream));
  return ARCB_OK;
}
