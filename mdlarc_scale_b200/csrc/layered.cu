// Layered models: the network is data (a list of mixers and feed-forwards).  Weight packing, cache and
// state layout, workspace, and the forward pass shared by prefill and the captured decode step.
//
// Padding: the residual width, the feed-forward width and the vocabulary are rounded up to 128 columns
// and every head to 64, 128 or 256; padded weights, gains and biases are zero, so padded columns carry
// exact zeros and every product meets the tensor-core tile sizes whatever the model's sizes are.  Latent attention
// pads the latent to 128 columns, the query latent, the rotated part and the heads to 64.
//
// A layer may run several times (loops); caches and states belong to a layer RUN, weights to a layer.
#include <cstring>

#include "attn_gqa.cuh"
#include "attn_latent.cuh"
#include "attn_prefill_gqa.cuh"
#include "engine.cuh"
#include "gemm.cuh"
#include "launch.cuh"
#include "layerops.cuh"
#include "mlstm.cuh"
#include "moe.cuh"

namespace {

int pad64(int v) { return (v + 63) / 64 * 64; }
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
  void* w_up = nullptr;        // [ffp][Wp]; gated: [2 ffp][Wp], 64 gate rows then the matching 64 up rows
  void* w_down = nullptr;      // [Wp][ffp]
  float* norm1b = nullptr;
  float* norm2b = nullptr;
  // latent attention
  int hp = 0;                  // heads, one zero head added where sections would not fill whole column tiles
  int panels() const { return (kvp + rotp) / 64; }   // of the cached rows
  int q_rankp = 0, kvp = 0, rotp = 0, n_down = 0, n_expand = 0, rot_table = 0;
  void* w_uq = nullptr;        // [hp * (dimp + rotp)][q_rankp]; w_proj holds [n_down][Wp]: query latent, latent, rotated part
  void* w_ukv = nullptr;       // [n_expand][kvp]: keys of all heads, then values of all heads
  void* w_ukt = nullptr;       // [hp * kvp][dimp]: the keys' rows transposed head by head
  float* dq_norm = nullptr;    // [q_rankp]
  float* dkv_norm = nullptr;   // [kvp]
  // mixture of experts
  int sffp = 0, n_router = 0;
  void* w_router = nullptr;    // [n_router][Wp]
  void* w_egu = nullptr;       // [experts][2 ffp][Wp]
  void* w_edown = nullptr;     // [experts][Wp][ffp]
  void* w_sgu = nullptr;       // [2 sffp][Wp]
  void* w_sdown = nullptr;     // [Wp][sffp]
};

// One pass of one layer.
struct LmRun {
  int layer;
  bool add_embed;              // the embedding joins x ahead of it
};

struct RotTable {
  int dims, pairs;
  double base;
};

}  // namespace

struct LayeredModel {
  arcb_model_desc d;
  int wp, vp, fmt, es;
  std::vector<LmLayer> layers;
  float* embed = nullptr;      // [vocab][Wp] fp32
  float* final_norm = nullptr;
  void* head = nullptr;        // [Vp][Wp]
  std::vector<LmRun> runs;
  std::vector<RotTable> rots;
  int n_proj_max = 0, n_proj32_max = 0, heads_max = 0, k_out_max = 0, ffp_max = 0;
  int cq_max = 0, lat_max = 0, expand_max = 0, n_wide_max = 0;   // query latent, heads x latent, expansion, residual-like outputs
  int window_max = 0;          // of the latent layers, 0: one sees everything
  int n_down_max = 0;          // fp32 projections of the latent layers
  bool has_moe = false;
  bool sandwich() const { return d.norm_place == ARCB_PLACE_SANDWICH; }
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
  std::vector<void*> k, v;     // per run: keys and values (its own or the shared layer's); latent rows in k
  std::vector<float*> S, n, m; // per run: recurrent state
  std::vector<float2*> rot;    // per rotation table
  float* y = nullptr;          // [R][Wp] a sublayer's output (sandwich norms)
  void* cq = nullptr;          // [R][q_rankp]
  void* qlat = nullptr;        // [lat_rows][hp * kvp]
  void* olat = nullptr;        // [lat_rows][hp * kvp]
  int lat_rows = 0;
  void* expand = nullptr;      // [expand_rows][n_expand]
  int expand_rows = 0;
  MoeArgs moe{};               // buffers
  void* moe_hid = nullptr;     // [max_slots][ffp]
  void* moe_out = nullptr;     // [max_slots][Wp]
  // the shared expert of a decode step runs beside the routed ones
  cudaStream_t side = nullptr;
  cudaEvent_t fork = nullptr, join = nullptr;
};

namespace {

struct LmWs {
  size_t x, xn, proj, proj32, gates, mix, hid, hn, logits, ascratch, gscratch, ints, y, cq, qlat, olat, total;
  size_t moe_z, moe_rows, moe_slots, moe_xs, moe_hid, moe_out;
  size_t n_ints;
  int head_rows, lat_rows, max_slots, max_rt;
};

// counts of every layer run with routed experts, and the number of tiles
size_t moe_ints(const LayeredModel& m) { return m.has_moe ? m.runs.size() * MOE_MAX_EXPERTS + 64 : 0; }

// Feed-forwards that go through the routed experts' buffers: the most slots and (row, choice) pairs of `rows` rows.
void moe_sizes(const LayeredModel& m, int rows, int* slots, int* rt, int* ffp, int* zp) {
  *slots = *rt = *ffp = *zp = 0;
  for (const LmLayer& L : m.layers)
    if (L.d.mlp == ARCB_MLP_MOE) {
      for (int gran = 128; gran <= 256; gran += 128) {
        const int s = arcb_moe_max_slots(rows, L.d.experts, L.d.top, gran);
        *slots = s > *slots ? s : *slots;
      }
      *rt = rows * L.d.top > *rt ? rows * L.d.top : *rt;
      *ffp = L.ffp > *ffp ? L.ffp : *ffp;
      *zp = L.n_router > *zp ? L.n_router : *zp;
    }
}

bool lm_tc(const LayeredModel& m) { return m.fmt != 2 && m.d.gemm_path != ARCB_GEMM_SIMT; }

// keys and values expanded for the tensor-core prefill attention
bool lm_expands(const LayeredModel& m, const LmLayer& L, int B, int T) {
  return L.d.mixer == ARCB_MIXER_LATENT && lm_tc(m) && m.d.attn_path == ARCB_ATTN_AUTO &&
         arcb_attn_prefill_latent_supported(L.dimp, L.rotp, L.vdimp, L.panels(), B, T, L.d.scale);
}
// Rows of the expansion scratch: enough for a block of queries with its window, and for about 16 k keys (more of
// them leave the L2 cache before they are read).
int lm_expand_rows(const LayeredModel& m, int B, int T) {
  bool any = false;
  for (const LmLayer& L : m.layers) any = any || lm_expands(m, L, B, T);
  if (!any) return 0;
  const int span = m.window_max > 0 && m.window_max < T ? m.window_max : T;
  const long long all = (long long)B * (pad128(T) + 128);
  return pad128(span + 256) + 128 + (int)(all < 16384 ? all : 16384);
}

int lm_latent_splits(const LmLayer& L, int B, int requested, int T) {
  if (requested > 0) return requested > 64 ? 64 : requested;
  const int keys = T > 0 && L.d.window > 0 && L.d.window < T ? L.d.window : T;
  return arcb_attn_latent_splits(B, L.hp, L.kvp, keys);
}

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

LmWs lm_ws(const LayeredModel& m, int B, int P, int splits, int requested) {
  const size_t R = (size_t)(B > P ? B : P);
  LmWs w;
  w.head_rows = B > 1024 ? B : (P < 1024 ? (P > B ? P : B) : 1024);
  size_t off = 0;
  auto take = [&](size_t bytes) { const size_t at = off; off = align_up(off + bytes, 1024); return at; };
  w.x = take(R * m.wp * 4);
  w.xn = take(R * m.wp * m.es);
  w.proj = take(R * m.n_proj_max * m.es);
  w.proj32 = take(R * (use_fused(m) ? m.n_down_max : m.n_proj32_max) * 4);
  w.gates = take(R * 2 * m.heads_max * 4);
  w.mix = take(R * m.k_out_max * m.es);
  w.hid = take(R * (size_t)m.ffp_max * m.es);
  w.hn = take((size_t)w.head_rows * m.wp * m.es);
  w.logits = take((size_t)w.head_rows * m.vp * 4);
  size_t asz = splits > 1 ? (size_t)B * m.heads_max * splits * (256 + 4) * 4 : 0;
  for (const LmLayer& L : m.layers)
    if (L.d.mixer == ARCB_MIXER_LATENT) {
      const int s = lm_latent_splits(L, B, requested, 0);
      const size_t need = s > 1 ? (size_t)B * L.hp * s * (L.kvp + 4) * 4 : 0;
      asz = need > asz ? need : asz;
    }
  w.ascratch = take(asz);
  w.gscratch = take(align_up((size_t)B, 128) * m.n_wide_max * 4);
  w.n_ints = (size_t)B * 7 + 64 + moe_ints(m);
  w.ints = take(w.n_ints * 4);
  w.y = take(m.sandwich() ? R * m.wp * 4 : 0);
  w.cq = take(R * (size_t)m.cq_max * m.es);
  // the queries in latent space exist for one slice of the rows at a time
  w.lat_rows = B > 2048 ? B : (int)(R < 2048 ? R : 2048);
  w.qlat = take((size_t)w.lat_rows * m.lat_max * m.es);
  w.olat = take((size_t)w.lat_rows * m.lat_max * m.es);
  int ffp, zp;
  moe_sizes(m, (int)R, &w.max_slots, &w.max_rt, &ffp, &zp);
  w.moe_z = take(R * (size_t)zp * 4);
  w.moe_rows = take((size_t)w.max_rt * 4 * 4);               // expert, place, weight, slot
  w.moe_slots = take(((size_t)w.max_slots + w.max_slots / 128 + 2) * 4);   // weights, experts of the tiles
  w.moe_xs = take((size_t)w.max_slots * m.wp * m.es * (m.has_moe ? 1 : 0));
  w.moe_hid = take((size_t)w.max_slots * ffp * m.es);
  w.moe_out = take((size_t)w.max_slots * m.wp * m.es * (m.has_moe ? 1 : 0));
  w.total = off;
  return w;
}

size_t kv_plane(const LayeredModel& m, const LmLayer& L, int B, int T, bool value) {
  return align_up((size_t)B * L.d.kv_heads * T * (value ? L.vdimp : L.dimp) * m.es, 1024);
}
size_t latent_plane(const LayeredModel& m, const LmLayer& L, int B, int T) {
  return align_up((size_t)B * T * (L.kvp + L.rotp) * m.es, 1024);
}
size_t rot_plane(const RotTable& r, int T) { return align_up((size_t)T * r.pairs * sizeof(float2), 1024); }
size_t expand_plane(const LayeredModel& m, int B, int T) {
  return align_up((size_t)lm_expand_rows(m, B, T) * m.expand_max * m.es, 1024);
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
    if (d.window < 0) return arcb_fail(ARCB_E_ARG, "window must not be negative");
    if (d.mixer == ARCB_MIXER_LATENT) {
      if (d.q_rank <= 0 || d.kv_rank <= 0 || d.rot_dim < 0 || d.rot_dims < 0 || d.rot_dims > d.rot_dim || d.rot_dims % 2)
        return arcb_fail(ARCB_E_ARG, "bad latent sizes");
      if (d.rot_dims > 0 && !(d.rot_base > 0.)) return arcb_fail(ARCB_E_ARG, "rot_base must be positive");
      if (d.kv_rank > 2048 || pad64(d.q_rank) + pad128(d.kv_rank) + pad64(d.rot_dim) > 6144)
        return arcb_fail(ARCB_E_UNSUPPORTED, "latents above 2048, or above 6144 columns with the query latent, are not implemented");
      if (d.qkv_bias || d.qk_norm || d.out_gate || d.q_temp_every || d.kv_from >= 0)
        return arcb_fail(ARCB_E_UNSUPPORTED, "latent attention has no biases, head norms, output gate, query gain or shared cache");
    } else if (d.dim > 256 || d.vdim > 256) {
      return arcb_fail(ARCB_E_UNSUPPORTED, "head sizes above 256 are not implemented");
    }
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
    } else if (d.mixer != ARCB_MIXER_LATENT) {
      return arcb_fail(ARCB_E_UNSUPPORTED, "unknown mixer");
    }
    if (d.mlp < ARCB_MLP_NONE || d.mlp > ARCB_MLP_MOE || (d.mlp != ARCB_MLP_NONE && d.d_ff <= 0) ||
        ((d.mlp == ARCB_MLP_GLU || d.mlp == ARCB_MLP_MOE) && d.glu != ARCB_GLU_SILU && d.glu != ARCB_GLU_CLAMPED))
      return arcb_fail(ARCB_E_UNSUPPORTED, "unknown feed-forward");
    if (d.mlp == ARCB_MLP_MOE) {
      if (md->norm_place != ARCB_PLACE_SANDWICH) return arcb_fail(ARCB_E_UNSUPPORTED, "routed experts need sandwich norms");
      if (d.experts <= 0 || d.top <= 0 || d.top > d.experts || d.shared_ff < 0) return arcb_fail(ARCB_E_ARG, "bad expert counts");
      if (d.experts > MOE_MAX_EXPERTS || d.top > MOE_MAX_TOP)
        return arcb_fail(ARCB_E_UNSUPPORTED, "more than 256 experts or 32 of them per token are not implemented");
    }
    if (md->loop_times != 1 && d.kv_from >= 0) return arcb_fail(ARCB_E_UNSUPPORTED, "layers of a looped model cannot share a cache");
  }
  if (md->norm_place != ARCB_PLACE_POST && md->norm_place != ARCB_PLACE_SANDWICH) return arcb_fail(ARCB_E_UNSUPPORTED, "unknown norm_place");
  if (md->norm_place == ARCB_PLACE_SANDWICH && (md->norm != ARCB_NORM_RMS || md->residual_alpha != 1.f))
    return arcb_fail(ARCB_E_UNSUPPORTED, "sandwich norms are RMS norms around an unweighted residual");
  if (md->loop_times < 1 || (md->loop_times > 1 && (md->loop_start < 0 || md->loop_stop > md->n_layers || md->loop_start >= md->loop_stop)))
    return arcb_fail(ARCB_E_ARG, "bad loop");
  if (md->loop_times > 1 && md->norm_place != ARCB_PLACE_SANDWICH) return arcb_fail(ARCB_E_UNSUPPORTED, "loops need sandwich norms");
  if (!arcb_device_ok()) return arcb_fail(ARCB_E_UNSUPPORTED, "current device is not compute capability 10.x");
  CKL(arcb_gemm_init(), "gemm init (shared-memory opt-in / cuTensorMapEncodeTiled lookup)");
  CKL(arcb_mlstm_chunk_init(), "chunkwise recurrence init (shared-memory opt-in)");
  CKL(arcb_attn_prefill_gqa_init(), "prefill attention init (shared-memory opt-in)");
  CKL(arcb_attn_latent_init(), "latent attention init (shared-memory opt-in)");
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
    const bool rec = d.mixer == ARCB_MIXER_MLSTM, latent = d.mixer == ARCB_MIXER_LATENT;
    L.dimp = latent ? pad64(d.dim) : pad_head(d.dim);
    L.vdimp = latent ? pad64(d.vdim) : pad_head(d.vdim);
    L.ffp = d.mlp == ARCB_MLP_NONE ? 0 : d.mlp == ARCB_MLP_RELU2 ? pad128(d.d_ff) : pad64(d.d_ff);
    L.own_kv = d.mixer == ARCB_MIXER_ATTENTION && d.kv_from < 0;
    L.hp = d.heads;
    if (latent) {
      L.q_rankp = pad64(d.q_rank);
      L.kvp = pad128(d.kv_rank);
      L.rotp = pad64(d.rot_dim > 0 ? d.rot_dim : 1);
      L.n_down = pad128(L.q_rankp + L.kvp + L.rotp);
      if (L.hp % 2 && ((L.dimp + L.rotp) % 128 || (L.dimp + L.vdimp) % 128 || L.vdimp % 128)) ++L.hp;
      L.n_expand = L.hp * (L.dimp + L.vdimp);
      L.rot_table = -1;
      if (d.rot_dims > 0) {
        for (size_t i = 0; i < m->rots.size(); ++i)
          if (m->rots[i].dims == d.rot_dims && m->rots[i].pairs == L.rotp / 2 && m->rots[i].base == d.rot_base) L.rot_table = (int)i;
        if (L.rot_table < 0) {
          L.rot_table = (int)m->rots.size();
          m->rots.push_back({d.rot_dims, L.rotp / 2, d.rot_base});
        }
      }
      const bool sees_all = d.window == 0 || (m->cq_max > 0 && m->window_max == 0);
      m->window_max = sees_all ? 0 : d.window > m->window_max ? d.window : m->window_max;
      m->cq_max = L.q_rankp > m->cq_max ? L.q_rankp : m->cq_max;
      m->lat_max = L.hp * L.kvp > m->lat_max ? L.hp * L.kvp : m->lat_max;
      m->expand_max = L.n_expand > m->expand_max ? L.n_expand : m->expand_max;
      m->n_down_max = L.n_down > m->n_down_max ? L.n_down : m->n_down_max;
    }
    L.k_out = L.hp * L.vdimp;
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
    L.n_proj = latent ? L.hp * (L.dimp + L.rotp) : pad128(at);   // latent: the queries
    r |= zalloc(e, &L.norm1, (size_t)m->wp * 4);
    r |= zalloc(e, &L.w_proj, (size_t)(latent ? L.n_down : L.n_proj) * m->wp * m->es);
    if (!latent) {
      r |= zalloc(e, &L.b_proj, (size_t)L.n_proj * 4);
      r |= zalloc(e, &L.q_norm, (size_t)L.dimp * 4);
      r |= zalloc(e, &L.k_norm, (size_t)L.dimp * 4);
      r |= zalloc(e, &L.head_norm, (size_t)L.k_out * 4);
    } else {
      r |= zalloc(e, &L.w_uq, (size_t)L.n_proj * L.q_rankp * m->es);
      r |= zalloc(e, &L.w_ukv, (size_t)L.n_expand * L.kvp * m->es);
      r |= zalloc(e, &L.w_ukt, (size_t)L.hp * L.kvp * L.dimp * m->es);
      r |= zalloc(e, &L.dq_norm, (size_t)L.q_rankp * 4);
      r |= zalloc(e, &L.dkv_norm, (size_t)L.kvp * 4);
    }
    r |= zalloc(e, &L.sink, (size_t)L.hp * 4);
    r |= zalloc(e, &L.w_out, (size_t)m->wp * L.k_out * m->es);
    if (m->sandwich()) r |= zalloc(e, &L.norm1b, (size_t)m->wp * 4);
    int hidden = 0;                // columns of the hidden buffer
    if (L.ffp) {
      r |= zalloc(e, &L.norm2, (size_t)m->wp * 4);
      if (m->sandwich()) r |= zalloc(e, &L.norm2b, (size_t)m->wp * 4);
      if (d.mlp == ARCB_MLP_MOE) {
        m->has_moe = true;
        L.n_router = pad128(d.experts);
        L.sffp = d.shared_ff > 0 ? pad64(d.shared_ff) : 0;
        hidden = L.sffp;
        r |= zalloc(e, &L.w_router, (size_t)L.n_router * m->wp * m->es);
        r |= zalloc(e, &L.w_egu, (size_t)d.experts * 2 * L.ffp * m->wp * m->es);
        r |= zalloc(e, &L.w_edown, (size_t)d.experts * m->wp * L.ffp * m->es);
        if (L.sffp) {
          r |= zalloc(e, &L.w_sgu, (size_t)2 * L.sffp * m->wp * m->es);
          r |= zalloc(e, &L.w_sdown, (size_t)m->wp * L.sffp * m->es);
        }
      } else {
        hidden = L.ffp;
        r |= zalloc(e, &L.w_up, (size_t)(d.mlp == ARCB_MLP_GLU ? 2 : 1) * L.ffp * m->wp * m->es);
        r |= zalloc(e, &L.w_down, (size_t)m->wp * L.ffp * m->es);
      }
    }
    m->n_proj_max = L.n_proj > m->n_proj_max ? L.n_proj : m->n_proj_max;
    const int n32 = latent ? L.n_down : L.n_proj;
    m->n_proj32_max = n32 > m->n_proj32_max ? n32 : m->n_proj32_max;
    m->heads_max = L.hp > m->heads_max ? L.hp : m->heads_max;
    m->k_out_max = L.k_out > m->k_out_max ? L.k_out : m->k_out_max;
    m->ffp_max = hidden > m->ffp_max ? hidden : m->ffp_max;
    m->layers.push_back(L);
  }
  m->n_wide_max = m->wp > m->n_down_max ? m->wp : m->n_down_max;
  for (int l = 0; l < md->n_layers; ++l) {
    if (md->loop_times > 1 && l == md->loop_start) {
      for (int t = 0; t < md->loop_times; ++t)
        for (int i = md->loop_start; i < md->loop_stop; ++i) m->runs.push_back({i, t > 0 && i == md->loop_start});
      l = md->loop_stop - 1;
    } else {
      m->runs.push_back({l, false});
    }
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
  // gate or up rows of a gated unit: blocks of 64, gates first
  auto gated = [&](void* p, int ff, bool up) {
    rows = ff; rb = 64; rbp = 128; row_off = up ? 64 : 0; cols = W; pitch = m.wp; dst = p;
  };
  const bool lat = L && L->d.mixer == ARCB_MIXER_LATENT, moe = L && L->d.mlp == ARCB_MLP_MOE;
  bool done = false;
  switch (kind) {
    case ARCB_L_EMBED: rows = m.d.vocab; cols = W; pitch = m.wp; dst = m.embed; weight = false; break;
    case ARCB_L_FINAL_NORM: vec(m.final_norm, W); break;
    case ARCB_L_HEAD: rows = m.d.vocab; cols = W; pitch = m.wp; dst = m.head; break;
    case ARCB_L_NORM1: vec(L->norm1, W); break;
    case ARCB_L_NORM2: if (L->ffp) vec(L->norm2, W); break;
    case ARCB_L_Q: if (!lat) rows_of(H, L->d.dim, L->dimp, L->off_q); break;
    case ARCB_L_Q_B: if (!lat) bias_of(H, L->d.dim, L->dimp, L->off_q); break;
    case ARCB_L_K: if (L->off_k >= 0) rows_of(nkv, L->d.dim, L->dimp, L->off_k); break;
    case ARCB_L_K_B: if (L->off_k >= 0) bias_of(nkv, L->d.dim, L->dimp, L->off_k); break;
    case ARCB_L_V: if (L->off_v >= 0) rows_of(nkv, L->d.vdim, L->vdimp, L->off_v); break;
    case ARCB_L_V_B: if (L->off_v >= 0) bias_of(nkv, L->d.vdim, L->vdimp, L->off_v); break;
    case ARCB_L_G: if (L->off_g >= 0) rows_of(H, L->d.vdim, L->vdimp, L->off_g); break;
    case ARCB_L_O: rows = W; cols = (long long)H * L->d.vdim; cb = L->d.vdim; cbp = L->vdimp; pitch = L->k_out; dst = L->w_out; break;
    case ARCB_L_Q_NORM: if (!lat) vec(L->q_norm, L->d.dim); break;
    case ARCB_L_K_NORM: if (!lat) vec(L->k_norm, L->d.dim); break;
    case ARCB_L_SINK: vec(L->sink, H); break;
    case ARCB_L_HEAD_NORM: if (!lat) vec(L->head_norm, (long long)H * L->d.vdim); cb = L->d.vdim; cbp = L->vdimp; break;
    case ARCB_L_I: if (rec) rows_of(1, H, H, L->off_gate); break;
    case ARCB_L_I_B: if (rec) bias_of(1, H, H, L->off_gate); break;
    case ARCB_L_F: if (rec) rows_of(1, H, H, L->off_gate + H); break;
    case ARCB_L_F_B: if (rec) bias_of(1, H, H, L->off_gate + H); break;
    case ARCB_L_UP:
      if (L->w_up && L->d.mlp == ARCB_MLP_GLU) { gated(L->w_up, L->d.d_ff, true); break; }
      if (L->w_up) { rows = L->d.d_ff; cols = W; pitch = m.wp; dst = L->w_up; }
      break;
    case ARCB_L_DOWN: if (L->w_down) { rows = W; cols = L->d.d_ff; pitch = L->ffp; dst = L->w_down; } break;
    case ARCB_L_GATE: if (L->w_up && L->d.mlp == ARCB_MLP_GLU) gated(L->w_up, L->d.d_ff, false); break;
    case ARCB_L_NORM1B: if (L->norm1b) vec(L->norm1b, W); break;
    case ARCB_L_NORM2B: if (L->norm2b) vec(L->norm2b, W); break;
    case ARCB_L_DQ: if (lat) { rows = L->d.q_rank; cols = W; pitch = m.wp; dst = L->w_proj; } break;
    case ARCB_L_DKV:
      if (lat) {      // the latent's rows, then the rotated part's, which start behind the latent's padding
        rows = L->d.kv_rank + L->d.rot_dim; rb = L->d.kv_rank; rbp = L->kvp; row_off = L->q_rankp; cols = W; pitch = m.wp; dst = L->w_proj;
        if (L->d.rot_dim > L->d.kv_rank) {
          CKL(arcb_launch_pack_blocks(src, dst, L->d.kv_rank, W, L->d.kv_rank, L->d.kv_rank, L->q_rankp, (int)W, (int)W, m.wp, m.fmt, stream), "pack_blocks");
          src += (size_t)L->d.kv_rank * W;
          numel -= (long long)L->d.kv_rank * W;
          rows = rb = rbp = L->d.rot_dim; row_off = L->q_rankp + L->kvp;
        }
      }
      break;
    case ARCB_L_DQ_NORM: if (lat) vec(L->dq_norm, L->d.q_rank); break;
    case ARCB_L_DKV_NORM: if (lat) vec(L->dkv_norm, L->d.kv_rank); break;
    case ARCB_L_UQ:
      if (lat) {      // head by head [unrotated, rotated]: two passes, as the two parts are padded apart
        const int hd = L->d.dim + L->d.rot_dim;
        rows = (long long)H * hd; cols = L->d.q_rank; pitch = L->q_rankp;
        if (numel != rows * cols) return arcb_fail(ARCB_E_ARG, "tensor has the wrong number of elements");
        for (int h = 0; h < H; ++h) {
          const float* hs = src + (size_t)h * hd * cols;
          const int at = h * (L->dimp + L->rotp);
          CKL(arcb_launch_pack_blocks(hs, L->w_uq, L->d.dim, cols, L->d.dim, L->d.dim, at, (int)cols, (int)cols, pitch, m.fmt, stream), "pack_blocks");
          if (L->d.rot_dim)
            CKL(arcb_launch_pack_blocks(hs + (size_t)L->d.dim * cols, L->w_uq, L->d.rot_dim, cols, L->d.rot_dim, L->d.rot_dim, at + L->dimp, (int)cols,
                                        (int)cols, pitch, m.fmt, stream), "pack_blocks");
        }
        done = true;
      }
      break;
    case ARCB_L_UK:
      if (lat) {
        rows = (long long)H * L->d.dim; rb = L->d.dim; rbp = L->dimp; cols = L->d.kv_rank; pitch = L->kvp; dst = L->w_ukv;
        if (numel == rows * cols)
          CKL(arcb_launch_pack_heads_t(src, L->w_ukt, H, L->d.dim, L->kvp, L->d.kv_rank, L->dimp, m.fmt, stream), "pack_heads");
      }
      break;
    case ARCB_L_UV:
      if (lat) {
        rows = (long long)H * L->d.vdim; rb = L->d.vdim; rbp = L->vdimp; row_off = L->hp * L->dimp; cols = L->d.kv_rank; pitch = L->kvp; dst = L->w_ukv;
      }
      break;
    case ARCB_L_ROUTER: if (moe) { rows = L->d.experts; cols = W; pitch = m.wp; dst = L->w_router; } break;
    case ARCB_L_EXPERT_GATE:
    case ARCB_L_EXPERT_UP:
      if (moe) {
        const long long per = (long long)L->d.d_ff * W;
        if (numel != per * L->d.experts) return arcb_fail(ARCB_E_ARG, "tensor has the wrong number of elements");
        for (int x = 0; x < L->d.experts; ++x)
          CKL(arcb_launch_pack_blocks(src + per * x, L->w_egu, L->d.d_ff, W, 64, 128, x * 2 * L->ffp + (kind == ARCB_L_EXPERT_UP ? 64 : 0), (int)W,
                                      (int)W, m.wp, m.fmt, stream), "pack_blocks");
        done = true;
      }
      break;
    case ARCB_L_EXPERT_DOWN:
      if (moe) { rows = (long long)L->d.experts * W; rb = (int)W; rbp = m.wp; cols = L->d.d_ff; pitch = L->ffp; dst = L->w_edown; }
      break;
    case ARCB_L_SHARED_GATE: if (L->w_sgu) gated(L->w_sgu, L->d.shared_ff, false); break;
    case ARCB_L_SHARED_UP: if (L->w_sgu) gated(L->w_sgu, L->d.shared_ff, true); break;
    case ARCB_L_SHARED_DOWN: if (L->w_sdown) { rows = W; cols = L->d.shared_ff; pitch = L->sffp; dst = L->w_sdown; } break;
  }
  if (done) {
    e->loaded[(size_t)kind * m.d.n_layers + layer] = 1;
    return ARCB_OK;
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
    bool ok = has(ARCB_L_NORM1, l) && has(ARCB_L_O, l);
    if (L.d.mixer == ARCB_MIXER_LATENT)
      ok = ok && has(ARCB_L_DQ, l) && has(ARCB_L_DQ_NORM, l) && has(ARCB_L_UQ, l) && has(ARCB_L_DKV, l) && has(ARCB_L_DKV_NORM, l) &&
           has(ARCB_L_UK, l) && has(ARCB_L_UV, l);
    else
      ok = ok && has(ARCB_L_Q, l);
    if (m.sandwich()) ok = ok && has(ARCB_L_NORM1B, l) && (!L.ffp || has(ARCB_L_NORM2B, l));
    if (rec || L.own_kv) ok = ok && has(ARCB_L_K, l) && has(ARCB_L_V, l);
    if (L.off_g >= 0) ok = ok && has(ARCB_L_G, l);
    if (rec) ok = ok && has(ARCB_L_I, l) && has(ARCB_L_I_B, l) && has(ARCB_L_F, l) && has(ARCB_L_F_B, l) && has(ARCB_L_HEAD_NORM, l);
    if (L.d.qkv_bias) ok = ok && has(ARCB_L_Q_B, l) && (!L.own_kv || (has(ARCB_L_K_B, l) && has(ARCB_L_V_B, l)));
    if (!rec && L.d.qk_norm) ok = ok && has(ARCB_L_Q_NORM, l) && (!L.own_kv || has(ARCB_L_K_NORM, l));
    if (!rec && L.d.sink) ok = ok && has(ARCB_L_SINK, l);
    if (L.ffp) ok = ok && has(ARCB_L_NORM2, l);
    if (L.ffp && L.d.mlp != ARCB_MLP_MOE) ok = ok && has(ARCB_L_UP, l) && has(ARCB_L_DOWN, l) && (L.d.mlp != ARCB_MLP_GLU || has(ARCB_L_GATE, l));
    if (L.ffp && L.d.mlp == ARCB_MLP_MOE)
      ok = ok && has(ARCB_L_ROUTER, l) && has(ARCB_L_EXPERT_GATE, l) && has(ARCB_L_EXPERT_UP, l) && has(ARCB_L_EXPERT_DOWN, l) &&
           (!L.sffp || (has(ARCB_L_SHARED_GATE, l) && has(ARCB_L_SHARED_UP, l) && has(ARCB_L_SHARED_DOWN, l)));
    if (!ok) return false;
  }
  return true;
}

// ---------------------------------------------------------------------------
// session
// ---------------------------------------------------------------------------
int64_t lm_cache_bytes(const arcb_engine* e, int B, int T) {
  const LayeredModel& m = *e->lm;
  size_t n = expand_plane(m, B, T);
  for (const RotTable& r : m.rots) n += rot_plane(r, T);
  for (const LmRun& run : m.runs) {
    const LmLayer& L = m.layers[run.layer];
    if (L.d.mixer == ARCB_MIXER_LATENT) n += latent_plane(m, L, B, T);
    if (L.own_kv) n += kv_plane(m, L, B, T, false) + kv_plane(m, L, B, T, true);
    if (L.d.mixer == ARCB_MIXER_MLSTM) n += st_plane(L, B, 0) + st_plane(L, B, 1) + st_plane(L, B, 2);
  }
  return (int64_t)(n ? n : 1024);
}

int64_t lm_workspace_bytes(const arcb_engine* e, int B, int P, int attn_splits) {
  return (int64_t)lm_ws(*e->lm, B, P, lm_splits(*e->lm, B, attn_splits, 0), attn_splits).total;
}

int lm_session_create(arcb_session* s) {
  const LayeredModel& m = *s->eng->lm;
  const arcb_session_desc& d = s->desc;
  const int B = d.n_seqs, T = d.t_max;
  LayeredSession* ls = new LayeredSession();
  s->ls = ls;
  ls->splits = lm_splits(m, B, d.attn_splits, T);
  const LmWs w = lm_ws(m, B, d.max_prefill_tokens, lm_splits(m, B, d.attn_splits, 0), d.attn_splits);
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
  ls->attn_scratch = reinterpret_cast<float*>(base + w.ascratch);
  ls->y = reinterpret_cast<float*>(base + w.y);
  ls->cq = base + w.cq;
  ls->qlat = base + w.qlat;
  ls->olat = base + w.olat;
  ls->lat_rows = w.lat_rows;
  ls->moe_hid = base + w.moe_hid;
  ls->moe_out = base + w.moe_out;
  MoeArgs& mo = ls->moe;
  mo.z = reinterpret_cast<float*>(base + w.moe_z);
  mo.max_slots = w.max_slots;
  mo.expert = reinterpret_cast<int*>(base + w.moe_rows);
  mo.rank = mo.expert + w.max_rt;
  mo.weight = reinterpret_cast<float*>(mo.rank + w.max_rt);
  mo.slot = mo.rank + 2 * (size_t)w.max_rt;
  mo.slot_weight = reinterpret_cast<float*>(base + w.moe_slots);
  mo.tile_expert = reinterpret_cast<int*>(mo.slot_weight + w.max_slots);
  mo.xs = base + w.moe_xs;
  ls->gemm_scratch = reinterpret_cast<float*>(base + w.gscratch);
  ls->head_rows = w.head_rows;
  ls->ints = reinterpret_cast<int*>(base + w.ints);
  ls->n_ints = w.n_ints;
  StepState& st = ls->st;
  st.n_seqs = B; st.t_max = T; st.max_new = d.max_new; st.stop_on_end = d.stop_on_end; st.end_token = d.end_token;
  int* p = ls->ints;
  st.cur_len = p; st.len0 = p + B; st.cur_tok = p + 2 * B; st.active = p + 3 * B; st.pos = p + 4 * B;
  st.kv_len = p + 5 * B; st.finished = p + 6 * B; st.n_finished = p + 7 * B;
  if (m.has_moe) {
    mo.count = p + 7 * B + 64;
    mo.n_tiles = mo.count + m.runs.size() * MOE_MAX_EXPERTS;
  }
  st.out_tokens = d.d_out_tokens; st.forced = d.d_forced; st.step_logits = d.d_step_logits;
  st.temperature = d.temperature; st.top_k = d.top_k; st.sample_seed = d.sample_seed; st.sample_stream = d.d_sample_stream;
  st.err = s->eng->d_err;
  uint8_t* c = reinterpret_cast<uint8_t*>(d.d_kv_cache);
  const size_t L = m.runs.size();
  ls->k.assign(L, nullptr); ls->v.assign(L, nullptr);
  ls->S.assign(L, nullptr); ls->n.assign(L, nullptr); ls->m.assign(L, nullptr);
  for (size_t l = 0; l < L; ++l) {
    const LmLayer& y = m.layers[m.runs[l].layer];
    if (y.d.mixer == ARCB_MIXER_LATENT) {
      ls->k[l] = c; c += latent_plane(m, y, B, T);
    } else if (y.own_kv) {
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
  for (const RotTable& r : m.rots) {
    ls->rot.push_back(reinterpret_cast<float2*>(c));
    c += rot_plane(r, T);
  }
  ls->expand = c;
  ls->expand_rows = lm_expand_rows(m, B, T);
  if (m.has_moe) {
    CK(cudaStreamCreateWithFlags(&ls->side, cudaStreamNonBlocking));
    CK(cudaEventCreateWithFlags(&ls->fork, cudaEventDisableTiming));
    CK(cudaEventCreateWithFlags(&ls->join, cudaEventDisableTiming));
  }
  return ARCB_OK;
}

void lm_session_destroy(LayeredSession* ls) {
  if (ls->fork) cudaEventDestroy(ls->fork);
  if (ls->join) cudaEventDestroy(ls->join);
  if (ls->side) cudaStreamDestroy(ls->side);
  delete ls;
}
int* lm_n_finished(arcb_session* s) { return s->ls->st.n_finished; }
bool lm_armed(const arcb_session* s) { return s->ls->armed; }

// ---------------------------------------------------------------------------
// forward pass
// ---------------------------------------------------------------------------
namespace {

int lm_gemm(const LayeredModel& m, const void* a, const void* w, GemmEpilogue& ep, int K, cudaStream_t stream, int variant = 0) {
  return arcb_launch_gemm(a, w, ep, K, m.fmt, lm_tc(m), stream, variant);
}

// Rows of one pass through the layers: a prefill call's packed tokens, or one row per sequence of a step.
struct Rows {
  int n;
  const int* pos;              // position of each row, < 0: held
  const int* seq;              // cache row, null: row index
  const int* kv_len;           // visible keys
  const arcb_prefill_args* pa; // null in a decode step
  const int* tokens;
};

// fp32 output of a product as it is, through the residual epilogue
int lm_store32(arcb_session* s, const void* a, const void* w, int K, int N, int rows, float* out, bool step, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  GemmEpilogue er{};
  er.mode = EPI_RESID; er.M = rows; er.N = N; er.x = out; er.overwrite = 1; er.act_f16 = m.fmt; er.err = s->eng->d_err;
  er.splitk_scratch = step && N <= m.n_wide_max ? s->ls->gemm_scratch : nullptr;
  CKL(lm_gemm(m, a, w, er, K, stream), "gemm");
  return ARCB_OK;
}

// the sublayer's last product: onto the residual stream, or to the buffer whose norm joins it
int lm_residual(arcb_session* s, const void* a, const void* w, int K, int rows, bool step, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  GemmEpilogue er{};
  er.mode = EPI_RESID; er.M = rows; er.N = m.wp; er.act_f16 = m.fmt; er.err = s->eng->d_err;
  er.x = m.sandwich() ? s->ls->y : s->ls->x;
  er.overwrite = m.sandwich() ? 1 : 0;
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

// Attention over cached latents.  A prompt's keys and values are expanded head by head for the tensor-core prefill
// kernel; in a decode step (and where that kernel does not apply) the queries move into the latent space instead.
int lm_latent(arcb_session* s, int l, const Rows& R, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  LayeredSession* ls = s->ls;
  const LmLayer& L = m.layers[m.runs[l].layer];
  const arcb_layer_desc& d = L.d;
  const int B = s->desc.n_seqs, T = s->desc.t_max, qh = L.dimp + L.rotp;
  const float2* rot = L.rot_table >= 0 ? ls->rot[L.rot_table] : nullptr;
  int r = lm_store32(s, ls->xn, L.w_proj, m.wp, L.n_down, R.n, ls->proj32, R.pa == nullptr, stream);
  if (r) return r;
  LatentPrepArgs p{};
  p.rows = R.n; p.pitch = L.n_down; p.q_rank = d.q_rank; p.q_rankp = L.q_rankp; p.kv_rank = d.kv_rank; p.kv_rankp = L.kvp;
  p.rot_dim = d.rot_dim; p.rotp = L.rotp; p.off_c = L.q_rankp; p.off_r = L.q_rankp + L.kvp; p.proj = ls->proj32;
  p.q_norm = L.dq_norm; p.kv_norm = L.dkv_norm; p.eps = m.d.norm_eps; p.rot = rot;
  p.cq = ls->cq; p.cache = ls->k[l]; p.pos = R.pos; p.seq = R.seq; p.t_max = T; p.n_seqs = B; p.fmt = m.fmt; p.err = s->eng->d_err;
  CKL(arcb_launch_latent_prep(p, stream), "latent prep");
  GemmEpilogue eq{};
  eq.mode = EPI_ACT; eq.M = R.n; eq.N = L.n_proj; eq.out16 = ls->proj; eq.act_f16 = m.fmt; eq.err = s->eng->d_err;
  if (rot) eq.rot = RotArgs{rot, R.pos, L.rotp / 2, qh, L.dimp, T};
  CKL(lm_gemm(m, ls->cq, L.w_uq, eq, L.q_rankp, stream), "query gemm");

  if (R.pa && R.pa->n_groups > 0 && lm_expands(m, L, B, T)) {
    const arcb_prefill_args& pa = *R.pa;
    for (int g = 0; g < pa.n_groups; ++g) {
      const int t0 = pa.h_group_tile[g], nt = pa.h_group_tile[g + 1] - t0, q0 = pa.h_group_qblock[g], nq = pa.h_group_qblock[g + 1] - q0;
      if (nt * 128 > ls->expand_rows) return arcb_fail(ARCB_E_ARG, "a group exceeds the expansion scratch");
      GemmEpilogue ek{};
      ek.mode = EPI_ACT; ek.M = nt * 128; ek.N = L.n_expand; ek.out16 = ls->expand; ek.act_f16 = m.fmt; ek.err = s->eng->d_err;
      ek.grp.tile_src = pa.d_tile_src + t0; ek.grp.panels = L.panels(); ek.grp.panel_rows = T; ek.grp.a_rows = (long long)B * L.panels() * T;
      CKL(lm_gemm(m, ls->k[l], L.w_ukv, ek, L.kvp, stream), "expansion gemm");
      AttnPrefillGqaArgs a{};
      a.q = ls->proj; a.q_pitch = L.n_proj; a.k = ls->expand; a.v = ls->expand; a.out = ls->mix; a.seq = R.seq; a.kv_count = R.kv_len;
      a.qblock_row0 = pa.d_qblock_row0 + q0; a.qblock_rows = pa.d_qblock_rows + q0; a.kv0 = pa.d_qblock_kv0 + q0; a.n_qblocks = nq;
      a.sink = d.sink ? L.sink : nullptr; a.n_rows = R.n; a.n_heads = a.n_kv = L.hp; a.dimp = L.dimp; a.vdimp = L.vdimp; a.t_max = T;
      a.n_seqs = B; a.window = d.window; a.kv_rows = nt * 128; a.kv_pitch = L.n_expand; a.v_col = L.hp * L.dimp; a.k_rot = ls->k[l];
      a.rotp = L.rotp; a.rot_panels = L.panels(); a.rot_panel = L.kvp / 64; a.scale = d.scale; a.act_f16 = m.fmt; a.err = s->eng->d_err;
      CKL(arcb_launch_attn_prefill_gqa(a, stream), "prefill attention");
    }
  } else {
    const uint8_t* q = reinterpret_cast<const uint8_t*>(ls->proj);
    for (int r0 = 0; r0 < R.n; r0 += ls->lat_rows) {
      const int n = R.n - r0 < ls->lat_rows ? R.n - r0 : ls->lat_rows;
      const void* qr = q + (size_t)r0 * L.n_proj * m.es;
      GemmEpilogue el{};
      el.mode = EPI_ACT; el.M = n; el.N = L.hp * L.kvp; el.out16 = ls->qlat; el.act_f16 = m.fmt; el.err = s->eng->d_err;
      el.grp.n_group = L.kvp; el.grp.a_group = qh; el.grp.lda = L.n_proj;
      CKL(lm_gemm(m, qr, L.w_ukt, el, L.dimp, stream), "latent query gemm");
      AttnLatentArgs a{};
      a.qlat = ls->qlat; a.q = qr; a.q_head = qh; a.q_off = L.dimp; a.cache = ls->k[l]; a.out = ls->olat;
      a.item_seq = R.seq ? R.seq + r0 : nullptr; a.item_len = R.kv_len + r0; a.sink = d.sink ? L.sink : nullptr; a.n_items = n; a.n_heads = L.hp;
      a.kvp = L.kvp; a.rotp = L.rotp; a.t_max = T; a.n_seqs = B; a.window = d.window; a.scale = d.scale; a.fmt = m.fmt; a.err = s->eng->d_err;
      a.n_splits = R.pa ? 1 : lm_latent_splits(L, B, s->desc.attn_splits, T);
      a.scratch = ls->attn_scratch;
      if (m.d.attn_path == ARCB_ATTN_AUTO && arcb_attn_latent_tc_supported(L.kvp, L.rotp, m.fmt, B, T, d.scale))
        CKL(arcb_launch_attn_latent_tc(a, stream), "latent attention");
      else
        CKL(arcb_launch_attn_latent_stream(a, stream), "latent attention");
      GemmEpilogue ev{};
      ev.mode = EPI_ACT; ev.M = n; ev.N = L.k_out; ev.act_f16 = m.fmt; ev.err = s->eng->d_err;
      ev.out16 = reinterpret_cast<uint8_t*>(ls->mix) + (size_t)r0 * L.k_out * m.es;
      ev.grp.n_group = L.vdimp; ev.grp.a_group = L.kvp; ev.grp.lda = L.hp * L.kvp;
      CKL(lm_gemm(m, ls->olat, reinterpret_cast<const uint8_t*>(L.w_ukv) + (size_t)L.hp * L.dimp * L.kvp * m.es, ev, L.kvp, stream), "value gemm");
    }
  }
  return lm_residual(s, ls->mix, L.w_out, L.k_out, R.n, R.pa == nullptr, stream);
}

// Feed-forward of layer run l from xn.  Routed experts leave their rows in ls->moe_out (joined by the norm that follows).
int lm_mlp(arcb_session* s, int l, const Rows& R, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  LayeredSession* ls = s->ls;
  const LmLayer& L = m.layers[m.runs[l].layer];
  const arcb_layer_desc& d = L.d;
  const bool step = R.pa == nullptr;
  GemmEpilogue eu{};
  eu.M = R.n; eu.out16 = ls->hid; eu.act_f16 = m.fmt; eu.err = s->eng->d_err;
  if (d.mlp == ARCB_MLP_RELU2) {
    eu.mode = EPI_RELU2; eu.N = L.ffp;
    CKL(lm_gemm(m, ls->xn, L.w_up, eu, m.wp, stream), "up gemm");
    return lm_residual(s, ls->hid, L.w_down, L.ffp, R.n, step, stream);
  }
  eu.mode = EPI_GLU;
  eu.glu.kind = d.glu;
  if (d.mlp == ARCB_MLP_GLU) {
    eu.N = 2 * L.ffp; eu.glu.limit = d.glu_limit;
    CKL(lm_gemm(m, ls->xn, L.w_up, eu, m.wp, stream), "gate/up gemm");
    return lm_residual(s, ls->hid, L.w_down, L.ffp, R.n, step, stream);
  }
  // the shared expert: of a decode step, whose launches leave most of the GPU idle, on a stream of its own
  if (L.sffp) {
    const bool beside = step && ls->side && !arcb_pdl_enabled();
    if (beside) {
      CK(cudaEventRecord(ls->fork, stream));
      CK(cudaStreamWaitEvent(ls->side, ls->fork, 0));
    }
    cudaStream_t st = beside ? ls->side : stream;
    eu.N = 2 * L.sffp; eu.glu.limit = d.shared_limit;
    CKL(lm_gemm(m, ls->xn, L.w_sgu, eu, m.wp, st), "shared gate/up gemm");
    const int r = lm_residual(s, ls->hid, L.w_sdown, L.sffp, R.n, step, st);
    if (r) return r;
    if (beside) CK(cudaEventRecord(ls->join, ls->side));
  }
  MoeArgs mo = ls->moe;
  mo.count += (size_t)l * MOE_MAX_EXPERTS;
  if (arcb_moe_router_inside(R.n, d.experts, m.wp, m.fmt)) {
    mo.z = nullptr;
    mo.w_router = L.w_router;
  } else {
    const int r = lm_store32(s, ls->xn, L.w_router, m.wp, L.n_router, R.n, const_cast<float*>(mo.z), false, stream);
    if (r) return r;
  }
  mo.rows = R.n; mo.experts = d.experts; mo.top = d.top; mo.z_pitch = L.n_router; mo.xn = ls->xn; mo.pitch = m.wp; mo.fmt = m.fmt;
  // pairs of row tiles (one expert each) once an expert fills them on average
  mo.gran = lm_tc(m) && arcb_gemm_max_pairs() > 0 && (long long)R.n * d.top >= 256ll * d.experts ? 256 : 128;
  CKL(arcb_launch_moe_route(mo, stream), "routing");
  const int slots = arcb_moe_max_slots(R.n, d.experts, d.top, mo.gran), variant = mo.gran == 256 ? 2 : 1;
  GemmEpilogue ee = eu;
  ee.M = slots; ee.N = 2 * L.ffp; ee.out16 = ls->moe_hid; ee.glu.limit = d.glu_limit; ee.glu.row = mo.slot_weight;
  ee.grp.tile_group = mo.tile_expert; ee.grp.n_tiles = mo.n_tiles; ee.grp.group_rows = 2 * L.ffp; ee.grp.w_rows = (long long)d.experts * 2 * L.ffp;
  CKL(lm_gemm(m, mo.xs, L.w_egu, ee, m.wp, stream, variant), "expert gate/up gemm");
  GemmEpilogue ed{};
  ed.mode = EPI_ACT; ed.M = slots; ed.N = m.wp; ed.out16 = ls->moe_out; ed.act_f16 = m.fmt; ed.err = s->eng->d_err;
  ed.grp.tile_group = mo.tile_expert; ed.grp.n_tiles = mo.n_tiles; ed.grp.group_rows = m.wp; ed.grp.w_rows = (long long)d.experts * m.wp;
  CKL(lm_gemm(m, ls->moe_hid, L.w_edown, ed, L.ffp, stream, variant), "expert down gemm");
  if (L.sffp && step && ls->side && !arcb_pdl_enabled()) CK(cudaStreamWaitEvent(stream, ls->join, 0));
  return ARCB_OK;
}

int lm_mixer(arcb_session* s, int l, const Rows& R, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  LayeredSession* ls = s->ls;
  const LmLayer& L = m.layers[m.runs[l].layer];
  const arcb_layer_desc& d = L.d;
  if (d.mixer == ARCB_MIXER_LATENT) return lm_latent(s, l, R, stream);
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
    a.window = d.window;
    CKL(arcb_launch_attn_prefill_gqa(a, stream), "prefill attention");
  } else {
    AttnGqaArgs a{};
    a.window = d.window;
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

// Sandwich norms: every sublayer reads the normed stream the one before it left in xn.
int lm_layers_sandwich(arcb_session* s, const Rows& R, float* residuals, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  LayeredSession* ls = s->ls;
  const int n_runs = (int)m.runs.size();
  LmNormArgs first{};
  first.kind = m.d.norm; first.rows = R.n; first.width = m.d.width; first.pitch = m.wp; first.fmt = m.fmt; first.eps = m.d.norm_eps;
  first.x_scale = 1.f; first.x = ls->x; first.w = m.layers[m.runs[0].layer].norm1; first.xn = ls->xn;
  CKL(arcb_launch_lm_norm(first, stream), "norm");
  for (int l = 0; l < n_runs; ++l) {
    const LmLayer& L = m.layers[m.runs[l].layer];
    const LmRun* next = l + 1 < n_runs ? &m.runs[l + 1] : nullptr;
    int r = lm_mixer(s, l, R, stream);
    if (r) return r;
    SandwichArgs a{};
    a.rows = R.n; a.width = m.d.width; a.pitch = m.wp; a.fmt = m.fmt; a.eps = m.d.norm_eps; a.x = ls->x; a.xn = ls->xn; a.y = ls->y;
    a.tokens = R.tokens; a.vocab = m.d.vocab;
    // what follows the layer's last sublayer
    auto last = [&]() {
      a.w_in = next ? m.layers[next->layer].norm1 : nullptr;
      a.embed = next && next->add_embed ? m.embed : nullptr;
      a.dense = residuals ? residuals + (size_t)l * R.n * m.d.width : nullptr;
    };
    a.w_out = L.norm1b;
    if (L.ffp) a.w_in = L.norm2;
    else last();
    CKL(arcb_launch_sandwich_norm(a, stream), "norm");
    if (!L.ffp) continue;
    r = lm_mlp(s, l, R, stream);
    if (r) return r;
    a.w_out = L.norm2b;
    if (L.d.mlp == ARCB_MLP_MOE) {
      a.ye = ls->moe_out; a.slot = ls->moe.slot; a.top = L.d.top;
      if (!L.sffp) a.y = nullptr;
    }
    last();
    CKL(arcb_launch_sandwich_norm(a, stream), "norm");
  }
  return ARCB_OK;
}

int lm_layers(arcb_session* s, const Rows& R, float* residuals, cudaStream_t stream) {
  const LayeredModel& m = *s->eng->lm;
  if (m.sandwich()) return lm_layers_sandwich(s, R, residuals, stream);
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
      r = lm_mlp(s, l, R, stream);
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
  a.embed = m.embed; a.alpha = m.d.residual_alpha; a.x = s->ls->x; a.xn = m.sandwich() ? nullptr : s->ls->xn;
  a.zero = s->ls->moe.count; a.n_zero = m.has_moe ? (int)(m.runs.size() * MOE_MAX_EXPERTS) : 0;
  return a;
}

// The integer state, and the cache: rows a query does not see are still operands of a product whose
// weights are zero, so they must hold finite numbers.
int lm_clear(arcb_session* s, cudaStream_t stream) {
  LayeredSession* ls = s->ls;
  if (ls->cleared) return ARCB_OK;
  CK(cudaMemsetAsync(ls->ints, 0, ls->n_ints * 4, stream));
  CK(cudaMemsetAsync(s->desc.d_kv_cache, 0, (size_t)lm_cache_bytes(s->eng, s->desc.n_seqs, s->desc.t_max), stream));
  const LayeredModel& m = *s->eng->lm;
  for (size_t i = 0; i < m.rots.size(); ++i)
    CKL(arcb_launch_rot_table(ls->rot[i], s->desc.t_max, m.rots[i].pairs, m.rots[i].dims, m.rots[i].base, stream), "rotation table");
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
  if (a->n_groups > 0 && (!a->h_group_qblock || !a->h_group_tile || !a->d_tile_src || !a->d_qblock_kv0 || a->n_qblocks <= 0))
    return arcb_fail(ARCB_E_ARG, "null group arrays");
  const Rows R{a->n_tokens, a->d_kv_slot, a->d_seq, a->d_kv_count, a, a->d_token_ids};
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
  const Rows R{B, ls->st.pos, nullptr, ls->st.kv_len, nullptr, ls->st.cur_tok};
  int r = lm_layers(s, R, nullptr, stream);
  if (r) return r;
  return lm_head(s, PICK_DECODE, B, nullptr, nullptr, nullptr, nullptr, stream);
}

extern "C" int arcb_session_expand_rows(arcb_session* s, int32_t* rows, int32_t* window) {
  if (!s || !s->ls || !rows || !window) return arcb_fail(ARCB_E_ARG, "arcb_session_expand_rows needs a layered session");
  const LayeredModel& m = *s->eng->lm;
  *rows = s->ls->expand_rows;
  *window = m.window_max > 0 && m.window_max < s->desc.t_max ? m.window_max : s->desc.t_max;
  return ARCB_OK;
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
