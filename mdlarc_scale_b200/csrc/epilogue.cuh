// GEMM epilogues shared by the tcgen05 and the CUDA-core GEMM kernels.
// Every epilogue consumes the accumulator in "quads": 4 consecutive output
// columns of one row, which is enough to keep RoPE pairs (2p, 2p+1) together.
#pragma once
#include "common.cuh"

enum : int {
  EPI_STORE_F32 = 0,  // y[m][n] = acc                               (tests)
  EPI_QKV_ROPE = 1,   // 3D RoPE on q,k; q -> q16, k/v -> KV cache    (src/inference.py:402-407)
  EPI_RESID = 2,      // x[m][n] += acc (+ bias[n])                   (src/inference.py:410-413)
  EPI_SWIGLU = 3,     // h16[m][j] = silu(g+bg) * (u+bu)              (src/transformer.py:446-449)
  EPI_RELU2 = 4,      // out[m][n] = relu(acc)^2 in the activation format
  EPI_HEADS = 5,      // fused mixer projection of a layered model (ProjArgs)
  EPI_ACT = 6,        // out[m][n] = acc in the activation format, optionally with rotated pairs (RotArgs)
  EPI_GLU = 7,        // out[m][j] = glu(s g, s u) in the activation format, s a factor of the row (GluArgs)
};

// Rotation of neighbouring column pairs of every head: head h owns columns [h * head, (h + 1) * head), its
// columns off + 2 i and off + 2 i + 1 (i < pairs) turn by the angle whose (cos, sin) is table[pos][i].  pairs covers
// all columns from off to the head's end; pairs that do not turn hold (1, 0).
struct RotArgs {
  const float2* table;   // [t_max][pairs], null: nothing turns
  const int* pos;        // [M], negative: position 0
  int pairs, head, off, t_max;
};

// Gated linear unit of a packed gate/up product (64 gate columns, then the 64 matching up columns).
struct GluArgs {
  int kind;              // ARCB_GLU_*
  float limit;           // ARCB_GLU_CLAMPED
  const float* row;      // [M] factor of both products, null: 1; a factor 0 yields 0 whatever the products are
};

// Products whose rows or columns belong to groups.  All fields zero: one plain product.
//   rows    : tile_src[t] is the A row of output rows [128 t, 128 t + 128) (null: 128 t); tile_group[t] picks the
//             rows [group * group_rows, ...) of W; n_tiles (device) is the number of tiles that hold anything
//   panels  : A is cut into panels of 64 columns, [sequence][panels][panel_rows][64]; tile_src then counts rows as
//             sequence * panel_rows + row
//   columns : columns [c n_group, (c + 1) n_group) read A columns [c a_group, c a_group + K)
struct GroupArgs {
  const int* tile_src;
  const int* tile_group;
  const int* n_tiles;
  int group_rows;
  long long w_rows;      // rows of W in all groups
  int n_group, a_group;
  int lda;               // row pitch of A in elements, 0: K
  long long a_rows;      // rows of A, 0: M (panels: of all panels)
  int panels, panel_rows;
};

// Fused projection of a mixer: the output columns are sections of whole heads, every head padded to
// 64, 128 or 256 columns (zero weights), every section starting at a multiple of 64 columns.
// q, the recurrence's k and v, and the output gate land at their own columns of `out` [M][N];
// attention keys and values go to the layer's cache rows; the recurrence's gates leave as fp32.
struct ProjArgs {
  int recurrent;         // 0 attention, 1 matrix-memory recurrence
  int M, N;
  int H, G;              // query heads, key/value heads
  int dim, dimp, vdim, vdimp;
  int off_q, off_k, off_v, off_g, off_gate;   // first column of each section, < 0: absent
  const float* bias;     // [N] or null
  const float* q_norm;   // [dimp] gains of the per-head RMS norm, null: no norm
  const float* k_norm;
  float eps, q_mul;      // q_mul: constant factor of the queries
  float temp_coef;       // query gain 1 + coef ln(floor((p + 1) / every) + 1); every 0: none
  int temp_every;
  const int* pos;        // [M] position of the row (its cache slot), < 0: the row stores nothing
  const int* seq;        // [M] cache row, null: row index
  void* kcache;          // [n_seqs][G][t_max][dimp] in the activation format
  void* vcache;          // [n_seqs][G][t_max][vdimp]
  int t_max, n_seqs;
  void* out;             // [M][N] activation format
  float* gates;          // [M][2 H]: biased pre-activations of the input gates, then of the forget gates
  int fmt;
  int* err;
};

__device__ __forceinline__ float sigmoid_f(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
__device__ __forceinline__ float sigmoid_exact(float x) { return 1.f / (1.f + expf(-x)); }

// gain of a query at position p
__device__ __forceinline__ float query_gain(const ProjArgs& a, int p) {
  float g = a.q_mul;
  if (a.temp_every > 0) g *= 1.f + a.temp_coef * logf((float)((p + 1) / a.temp_every) + 1.f);
  return g;
}
// cache row of (row m, key/value head 0), or -1 when the row stores nothing
__device__ __forceinline__ long long proj_cache_row(const ProjArgs& a, int m) {
  const int s = a.pos[m], b = a.seq ? a.seq[m] : m;
  if (s < 0) return -1;
  if (s >= a.t_max || b < 0 || b >= a.n_seqs) {
    arcb_set_error(a.err, ARCB_DEV_BAD_INDEX);
    return -1;
  }
  return (long long)b * a.G * a.t_max + s;
}

struct GemmEpilogue {
  int mode;
  int M, N;      // GEMM output extent (N counts packed columns for EPI_SWIGLU)
  int act_f16;   // format of 16-bit outputs (q16 / h16)
  float* y;      // EPI_STORE_F32: [M][N]
  float* x;      // EPI_RESID: residual stream [M][N], updated in place
  const float* bias;  // EPI_RESID: [N] or null; EPI_SWIGLU: [N] packed like the weight rows
  float* splitk_scratch;  // EPI_RESID, optional: >= 128 * ceil(M / 128) * N floats; allows the split-K kernel for few-row launches
  void* out16;   // EPI_QKV_ROPE: q16 [M][d]; EPI_SWIGLU: h16 [M][N/2]
  // EPI_QKV_ROPE
  const int* pos;   // [M][3] raw (x, y, z); clamped here like RotaryEmbedding3D.apply_rotary
  const int* slot;  // [M] cache position of the row's K/V, < 0: do not store
  const int* seq;   // [M] cache row (sequence) of the token; null = row index
  __nv_bfloat16* kcache;  // layer K base [B][H][t_max][64]
  __nv_bfloat16* vcache;  // layer V base
  void* k16;              // optional [n_kv_rows][d]: K of this call in the activation format
  void* v16;              //   (operands of the tensor-core prefill attention)
  const int* kv_row;      // [M] row of k16/v16 for this token, < 0: none
  int kv16_rows;          // rows of k16 / v16
  int kv16_identity;      // kv_row[m] == m for m < kv16_rows and < 0 after: rows can be stored as boxes
  int t_max, n_heads, d_model, n_seqs;
  const float* rope;  // cos_x | sin_x | cos_y | sin_y | cos_z | sin_z
  int max_x, max_y, max_z;
  int* err;           // error word; word 1 counts 16-bit saturations
  ProjArgs pj;        // EPI_HEADS
  int overwrite;      // EPI_RESID: x = acc instead of x += acc
  RotArgs rot;        // EPI_ACT
  GluArgs glu;        // EPI_GLU
  GroupArgs grp;
};

struct RopeRow {
  int x, y, z;
  long long kv_row;  // (seq * H) * t_max + slot, or -1
  int row16;         // row of k16/v16, or -1
};

__device__ __forceinline__ RopeRow rope_row_ctx(const GemmEpilogue& e, int m) {
  RopeRow r;
  r.row16 = (e.k16 && e.kv_row) ? e.kv_row[m] : -1;
  const int px = e.pos[3 * m + 0], py = e.pos[3 * m + 1], pz = e.pos[3 * m + 2];
  r.x = min(max(px, 0), e.max_x - 1);
  r.y = min(max(py, 0), e.max_y - 1);
  r.z = min(max(pz, 0), e.max_z - 1);
  const int s = e.slot[m];
  const int b = e.seq ? e.seq[m] : m;
  if (s < 0) {
    r.kv_row = -1;
  } else if (s >= e.t_max || b < 0 || b >= e.n_seqs) {
    arcb_set_error(e.err, ARCB_DEV_BAD_INDEX);
    r.kv_row = -1;
  } else {
    r.kv_row = ((long long)b * e.n_heads) * e.t_max + s;
  }
  return r;
}

// cos/sin of rotary pair p (0..31) at the row's clamped position.
__device__ __forceinline__ float2 rope_cs(const GemmEpilogue& e, const RopeRow& r, int p) {
  const float* t = e.rope;
  const int nx = e.max_x * ARCB_ROPE_PX, ny = e.max_y * ARCB_ROPE_PY, nz = e.max_z * ARCB_ROPE_PZ;
  int ic;
  if (p < ARCB_ROPE_PX) {
    ic = r.x * ARCB_ROPE_PX + p;
    return make_float2(__ldg(t + ic), __ldg(t + nx + ic));
  } else if (p < ARCB_ROPE_PX + ARCB_ROPE_PY) {
    ic = r.y * ARCB_ROPE_PY + (p - ARCB_ROPE_PX);
    return make_float2(__ldg(t + 2 * nx + ic), __ldg(t + 2 * nx + ny + ic));
  }
  ic = r.z * ARCB_ROPE_PZ + (p - ARCB_ROPE_PX - ARCB_ROPE_PY);
  return make_float2(__ldg(t + 2 * nx + 2 * ny + ic), __ldg(t + 2 * nx + 2 * ny + nz + ic));
}

// out[2p] = v[2p] cos - v[2p+1] sin ; out[2p+1] = v[2p+1] cos + v[2p] sin
// (src/transformer.py:51-58, 184-185)
__device__ __forceinline__ void epi_qkv_quad(const GemmEpilogue& e, const RopeRow& r, int m, int n,
                                             float4 v) {
  const int d = e.d_model;
  const int sec = n / d;           // 0 q, 1 k, 2 v
  const int c = n - sec * d;       // column inside the section
  const int h = c >> 6, dim = c & 63;
  if (sec < 2) {
    const int p = dim >> 1;
    const float2 cs0 = rope_cs(e, r, p), cs1 = rope_cs(e, r, p + 1);
    float4 o;
    o.x = v.x * cs0.x - v.y * cs0.y;
    o.y = v.y * cs0.x + v.x * cs0.y;
    o.z = v.z * cs1.x - v.w * cs1.y;
    o.w = v.w * cs1.x + v.z * cs1.y;
    v = o;
  }
  if (sec == 0) {
    uint2 pk;
    pk.x = pack2_act_chk(v.x, v.y, e.act_f16, e.err);
    pk.y = pack2_act_chk(v.z, v.w, e.act_f16, e.err);
    *reinterpret_cast<uint2*>(reinterpret_cast<uint16_t*>(e.out16) + (size_t)m * d + c) = pk;
  } else {
    if (r.kv_row >= 0) {
      __nv_bfloat16* base = (sec == 1) ? e.kcache : e.vcache;
      const long long row = r.kv_row + (long long)h * e.t_max;
      uint2 pk;
      pk.x = pack2_bf16(v.x, v.y);
      pk.y = pack2_bf16(v.z, v.w);
      *reinterpret_cast<uint2*>(base + row * ARCB_HEAD_DIM + dim) = pk;
    }
    if (r.row16 >= 0) {
      uint16_t* base16 = reinterpret_cast<uint16_t*>((sec == 1) ? e.k16 : e.v16);
      uint2 pk;
      pk.x = pack2_act_chk(v.x, v.y, e.act_f16, e.err);
      pk.y = pack2_act_chk(v.z, v.w, e.act_f16, e.err);
      *reinterpret_cast<uint2*>(base16 + (size_t)r.row16 * d + c) = pk;
    }
  }
}

// Rotate the 16 rotary pairs [P0, P0 + 16) held in v[0..32) (P0 is 0 or 16: first or second half of
// a 64-wide head).  Which table a pair uses (x: pairs 0-9, y: 10-19, z: 20-31) is known at compile
// time, so the loop unrolls into straight table loads.
template <int P0>
__device__ __forceinline__ void rope_rotate32(const GemmEpilogue& e, const RopeRow& r, float (&v)[32]) {
  const int nx = e.max_x * ARCB_ROPE_PX, ny = e.max_y * ARCB_ROPE_PY, nz = e.max_z * ARCB_ROPE_PZ;
  const float* cx = e.rope + r.x * ARCB_ROPE_PX;
  const float* sx = cx + nx;
  const float* cy = e.rope + 2 * nx + r.y * ARCB_ROPE_PY;
  const float* sy = cy + ny;
  const float* cz = e.rope + 2 * nx + 2 * ny + r.z * ARCB_ROPE_PZ;
  const float* sz = cz + nz;
#pragma unroll
  for (int i = 0; i < 16; ++i) {
    constexpr int PX = ARCB_ROPE_PX, PXY = ARCB_ROPE_PX + ARCB_ROPE_PY;
    const int p = P0 + i;
    float c, s;
    if (p < PX) { c = __ldg(cx + p); s = __ldg(sx + p); }
    else if (p < PXY) { c = __ldg(cy + (p - PX)); s = __ldg(sy + (p - PX)); }
    else { c = __ldg(cz + (p - PXY)); s = __ldg(sz + (p - PXY)); }
    const float a = v[2 * i], b = v[2 * i + 1];
    v[2 * i] = a * c - b * s;
    v[2 * i + 1] = b * c + a * s;
  }
}

// 32 consecutive QKV output columns [n0, n0 + 32) of row m (n0 % 32 == 0: one half of one head of
// one of the q / k / v sections): RoPE on q and k, then 16-byte stores of q16 or of the bf16 cache
// row (+ the call's 16-bit K/V scratch row).
__device__ __forceinline__ void epi_qkv_chunk32(const GemmEpilogue& e, const RopeRow& r, int m, int n0,
                                                const uint32_t (&acc)[32]) {
  const int d = e.d_model;
  const int sec = n0 / d;
  const int c = n0 - sec * d;
  const int h = c >> 6, dim0 = c & 63;
  float v[32];
#pragma unroll
  for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(acc[i]);
  if (sec < 2) {
    if (dim0 == 0) rope_rotate32<0>(e, r, v);
    else rope_rotate32<16>(e, r, v);
  }
  if (sec == 0) {
    uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<uint16_t*>(e.out16) + (size_t)m * d + c);
#pragma unroll
    for (int q = 0; q < 4; ++q)
      dst[q] = make_uint4(pack2_act_chk(v[8 * q], v[8 * q + 1], e.act_f16, e.err), pack2_act_chk(v[8 * q + 2], v[8 * q + 3], e.act_f16, e.err),
                          pack2_act_chk(v[8 * q + 4], v[8 * q + 5], e.act_f16, e.err), pack2_act_chk(v[8 * q + 6], v[8 * q + 7], e.act_f16, e.err));
    return;
  }
  if (r.kv_row >= 0) {
    __nv_bfloat16* base = (sec == 1) ? e.kcache : e.vcache;
    uint4* dst = reinterpret_cast<uint4*>(base + (r.kv_row + (long long)h * e.t_max) * ARCB_HEAD_DIM + dim0);
#pragma unroll
    for (int q = 0; q < 4; ++q)
      dst[q] = make_uint4(pack2_bf16(v[8 * q], v[8 * q + 1]), pack2_bf16(v[8 * q + 2], v[8 * q + 3]),
                          pack2_bf16(v[8 * q + 4], v[8 * q + 5]), pack2_bf16(v[8 * q + 6], v[8 * q + 7]));
  }
  if (r.row16 >= 0) {
    uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<uint16_t*>((sec == 1) ? e.k16 : e.v16) +
                                          (size_t)r.row16 * d + c);
#pragma unroll
    for (int q = 0; q < 4; ++q)
      dst[q] = make_uint4(pack2_act_chk(v[8 * q], v[8 * q + 1], e.act_f16, e.err), pack2_act_chk(v[8 * q + 2], v[8 * q + 3], e.act_f16, e.err),
                          pack2_act_chk(v[8 * q + 4], v[8 * q + 5], e.act_f16, e.err), pack2_act_chk(v[8 * q + 6], v[8 * q + 7], e.act_f16, e.err));
  }
}

__device__ __forceinline__ void epi_resid_quad(const GemmEpilogue& e, int m, int n, float4 v) {
  float4* px = reinterpret_cast<float4*>(e.x + (size_t)m * e.N + n);
  float4 r = e.overwrite ? make_float4(0.f, 0.f, 0.f, 0.f) : *px;
  if (e.bias) {
    const float4 b = __ldg(reinterpret_cast<const float4*>(e.bias + n));
    v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
  }
  r.x += v.x; r.y += v.y; r.z += v.z; r.w += v.w;
  *px = r;
}

__device__ __forceinline__ void epi_store_quad(const GemmEpilogue& e, int m, int n, float4 v) {
  *reinterpret_cast<float4*>(e.y + (size_t)m * e.N + n) = v;
}

__device__ __forceinline__ float relu2_f(float v) { v = fmaxf(v, 0.f); return v * v; }

__device__ __forceinline__ void epi_relu2_quad(const GemmEpilogue& e, int m, int n, float4 v) {
  v = make_float4(relu2_f(v.x), relu2_f(v.y), relu2_f(v.z), relu2_f(v.w));
  if (e.act_f16 == 1 && fmaxf(fmaxf(v.x, v.y), fmaxf(v.z, v.w)) > 65504.f) arcb_count_saturation(e.err);
  st_act4(e.out16, (size_t)m * e.N + n, v, e.act_f16);
}

__device__ __forceinline__ float silu_f(float g) { return __fdividef(g, 1.f + __expf(-g)); }

// Packed column n (n % 128 < 64) holds gate outputs, n + 64 the matching up outputs.
__device__ __forceinline__ void epi_swiglu_quad(const GemmEpilogue& e, int m, int n, float4 g,
                                                float4 u) {
  if (e.bias) {
    const float4 bg = __ldg(reinterpret_cast<const float4*>(e.bias + n));
    const float4 bu = __ldg(reinterpret_cast<const float4*>(e.bias + n + 64));
    g.x += bg.x; g.y += bg.y; g.z += bg.z; g.w += bg.w;
    u.x += bu.x; u.y += bu.y; u.z += bu.z; u.w += bu.w;
  }
  const int j = (n >> 7) * 64 + (n & 127);
  uint2 pk;
  pk.x = pack2_act_chk(silu_f(g.x) * u.x, silu_f(g.y) * u.y, e.act_f16, e.err);
  pk.y = pack2_act_chk(silu_f(g.z) * u.z, silu_f(g.w) * u.w, e.act_f16, e.err);
  *reinterpret_cast<uint2*>(reinterpret_cast<uint16_t*>(e.out16) + (size_t)m * (e.N >> 1) + j) = pk;
}

// first A row of a row tile
__device__ __forceinline__ int group_a_row(const GroupArgs& g, int tile) {
  if (!g.tile_src) return tile * 128;
  const int r = g.tile_src[tile];
  return g.panels ? r + r / g.panel_rows * (g.panels - 1) * g.panel_rows : r;
}

// ---- EPI_ACT ----
// (cos, sin) row of the position of row m
__device__ __forceinline__ const float2* rot_row(const GemmEpilogue& e, int m) {
  const int p = min(max(e.rot.pos[m], 0), e.rot.t_max - 1);
  return e.rot.table + (size_t)p * e.rot.pairs;
}
// two neighbouring pairs by (cos, sin, cos, sin)
__device__ __forceinline__ float4 rotate4(float4 v, float4 a) {
  return make_float4(v.x * a.x - v.y * a.y, v.y * a.x + v.x * a.y, v.z * a.z - v.w * a.w, v.w * a.z + v.z * a.w);
}
// columns n .. n + 3 (n % 4 == 0) of a row whose table row is cs
__device__ __forceinline__ float4 rot_quad(const GemmEpilogue& e, const float2* cs, int n, float4 v) {
  const int c = n % e.rot.head - e.rot.off;
  if (c < 0) return v;
  return rotate4(v, __ldg(reinterpret_cast<const float4*>(cs + (c >> 1))));
}
__device__ __forceinline__ void epi_act_quad(const GemmEpilogue& e, int m, int n, float4 v) {
  if (e.rot.table) v = rot_quad(e, rot_row(e, m), n, v);
  if (e.act_f16 == 1 && fmaxf(fmaxf(fabsf(v.x), fabsf(v.y)), fmaxf(fabsf(v.z), fabsf(v.w))) > 65504.f) arcb_count_saturation(e.err);
  st_act4(e.out16, (size_t)m * e.N + n, v, e.act_f16);
}

// ---- EPI_GLU ----
// EXACT: the accurate exponential and division (32-bit models), else the fast ones.
template <bool EXACT>
__device__ __forceinline__ float glu_sigmoid(float x) {
  return EXACT ? 1.f / (1.f + expf(-x)) : __fdividef(1.f, 1.f + __expf(-x));
}
template <bool EXACT>
__device__ __forceinline__ float glu_f(const GluArgs& a, float s, float g, float u) {
  if (s == 0.f) return 0.f;
  g *= s;
  u *= s;
  if (a.kind == 1) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit);
    return g * glu_sigmoid<EXACT>(1.702f * g) * (u + 1.f);
  }
  return g * glu_sigmoid<EXACT>(g) * u;
}
__device__ __forceinline__ void epi_glu_quad(const GemmEpilogue& e, int m, int n, float4 g, float4 u) {
  const float s = e.glu.row ? e.glu.row[m] : 1.f;
  const size_t at = (size_t)m * (e.N >> 1) + (n >> 7) * 64 + (n & 127);
  float4 v;
  if (e.act_f16 == 2) {
    v = make_float4(glu_f<true>(e.glu, s, g.x, u.x), glu_f<true>(e.glu, s, g.y, u.y), glu_f<true>(e.glu, s, g.z, u.z),
                    glu_f<true>(e.glu, s, g.w, u.w));
  } else {
    v = make_float4(glu_f<false>(e.glu, s, g.x, u.x), glu_f<false>(e.glu, s, g.y, u.y), glu_f<false>(e.glu, s, g.z, u.z),
                    glu_f<false>(e.glu, s, g.w, u.w));
    if (e.act_f16 == 1 && fmaxf(fmaxf(fabsf(v.x), fabsf(v.y)), fmaxf(fabsf(v.z), fabsf(v.w))) > 65504.f) arcb_count_saturation(e.err);
  }
  st_act4(e.out16, at, v, e.act_f16);
}
