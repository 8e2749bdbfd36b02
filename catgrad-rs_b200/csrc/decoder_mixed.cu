// decoder_mixed.cu — decoders whose layers carry different sequence mixers and may run in a loop:
// their weights, per-sequence caches and states, and the walk over their layers.  The entry points
// (prefill, append, decode with its captured graph, generate) are those of decoder.cu.
//
// A sequence lives in a slot.  Per layer run (a looped layer counts once per pass, a layer with another
// one's parameters is a run of that layer) a slot holds
//   attention          [kv heads, max_seq, head size] keys and values
//   latent attention   [max_seq, Lw] cached rows (normed latent, rotated key part)
//   delta, ssd         an f32 matrix per head and the last inputs of the convolutions
//   lightning, gla     an f32 matrix per head
//   lru                an f32 value per channel and the last inputs of the convolution
// (of two mixers side by side, both their parts).
// Nothing is cleared when a slot is reused: a row whose first position is 0 starts from zeros.
// Batches are rows of unequal length, packed token after token; every kernel finds a token's row,
// slot and position through the row tables (RowsDev).  In a decode step the tables stay as they
// are and a device counter moves all positions, so the step is one CUDA graph.
//
// Fused steps: all projections of a mixer, or of two side by side, are one GEMM (w_in), their two output
// projections one more with their sum (w_o); a post-norm, the residual add and
// the next pre-norm are one pass (k_row_update), which also writes the two-part rows a looped
// input reads and takes the sum over a token's experts.  Factors on norms' results and on a mixer's
// gains are folded into the f32 gains.  Without post-norms that pass is k_stream_update: the weighted sum over a token's
// experts, the mixing of the residual streams (a plain residual stream is one stream with unit
// coefficients), the next sublayer's input and its norm.  Matrices are padded with zeros to multiples
// of 8 (attention heads to the sizes of its tensor-core kernels) where the tensor cores want it.

#include <algorithm>
#include <cmath>
#include <cstring>

#include "decoder.h"
#include "mixers.h"

namespace cg {

namespace {
inline int64_t up8(int64_t n) { return (n + 7) / 8 * 8; }
inline int64_t up16(int64_t n) { return (n + 15) / 16 * 16; }
}  // namespace

struct MixedLayer {
  cg_layer_config k{};
  std::vector<double> decay;            // lightning
  std::unique_ptr<MixedLayer> beside;   // a second mixer: its mixer's members only
  int64_t in_row = 0, out_col = 0;      // where this mixer starts in w_in (rows) and w_o (columns), which both share
  cg_tensor *n1 = nullptr, *n1b = nullptr, *n2 = nullptr, *n2b = nullptr;
  cg_tensor *n1b_bias = nullptr, *n2b_bias = nullptr, *n1_bias = nullptr, *n2_bias = nullptr;
  cg_tensor *w_in = nullptr, *w_o = nullptr, *w_gu = nullptr, *w_down = nullptr;
  int64_t Np = 0;       // columns of the projection
  int64_t Fp = 0;       // padded feed-forward width
  int Do = 0;           // columns a head takes in the mixer's output
  int64_t Ko = 0;       // width of the mixer's output
  // coefficients of the streams, per sublayer
  cg_tensor *hc_in[2] = {nullptr, nullptr}, *hc_out[2] = {nullptr, nullptr}, *hc_mix[2] = {nullptr, nullptr};
  // experts, stacked
  cg_tensor *router = nullptr, *correction = nullptr, *we_gate = nullptr, *we_up = nullptr, *we_down = nullptr;
  int64_t Fd = 0;       // padded width of w_gu: the dense feed-forward or the shared expert, 0 = neither
  cg_tensor *up_bias = nullptr, *down_bias = nullptr;
  // sublayers side by side: norms of two mixers' results, weights of the depth average, the token's input
  cg_tensor *out_gain = nullptr, *average = nullptr, *side_gate = nullptr, *side_proj = nullptr, *side_norm = nullptr;
  int64_t ff_col = -1;  // >= 0: the feed-forward's units are columns of the mixer's output, w_down part of w_o
  // attention
  cg_tensor *q_gain = nullptr, *k_gain = nullptr, *sink = nullptr, *q_temp = nullptr, *bias = nullptr;
  int Dk = 0, Dv = 0;   // columns a key and a value head take
  // latent attention
  cg_tensor *c_gain = nullptr, *uk = nullptr, *uv = nullptr, *w_kv = nullptr, *cos_t = nullptr, *sin_t = nullptr;
  int64_t Lw = 0;       // width of a cached row
  int dkv_off = 0, Dq = 0;
  // recurrences
  cg_tensor *conv_w = nullptr, *conv_b = nullptr, *a_log = nullptr, *dt_bias = nullptr, *dskip = nullptr, *norm = nullptr,
            *log_decay = nullptr, *coef = nullptr, *w_a2 = nullptr, *w_g2 = nullptr;
  cg_tensor *ra = nullptr, *ri = nullptr, *ra_b = nullptr, *ri_b = nullptr, *xb = nullptr, *yb = nullptr;  // lru
  int zs = 0, a1_off = 0, g1_off = 0, a_rank = 0, g_rank = 0, x_off = 0;
  bool chunked = false;  // prompts run on the tensor cores, 64 tokens at a time
  int H = 0, KH = 0, dk = 0, dv = 0, dvs = 0, C = 0, gate_off = 0, small_off = 0, q_off = 0, k_off = 0, v_off = 0, qs = 0, vs = 0;

  bool lru() const { return k.mixer == CG_MIX_LRU; }
  bool key_decay() const { return k.mixer == CG_MIX_CHANNEL_DELTA || k.mixer == CG_MIX_GLA; }
  bool delta() const { return k.mixer == CG_MIX_DELTA || k.mixer == CG_MIX_CHANNEL_DELTA; }
  bool recurrent() const { return delta() || lru() || k.mixer == CG_MIX_SSD || k.mixer == CG_MIX_LIGHTNING || k.mixer == CG_MIX_GLA; }
  float out_scale() const { return k.out_scale != 0. ? (float)k.out_scale : 1.f; }
  int64_t in_width() const { return Np + (beside ? beside->Np : 0); }
  int64_t out_width() const { return Ko + (beside ? beside->Ko : 0) + (ff_col >= 0 ? Fd : 0); }
};

struct MixedRun {
  int layer;
  bool starts_pass;
  cg_tensor *cache = nullptr;                  // latent attention; keys of attention
  cg_tensor *cache_v = nullptr;                // attention
  cg_tensor *state = nullptr, *tail = nullptr;  // recurrences
  std::unique_ptr<MixedRun> beside;             // of the second mixer
};

struct MixedModel {
  std::vector<MixedLayer> layers;
  std::vector<MixedRun> runs;
  bool loop = false;        // passes start from w_loop
  bool f32 = false;
  bool sandwich = false;    // norms behind the sublayers too (k_row_update); else streams (k_stream_update)
  bool parallel = false;    // the sublayers of a layer run side by side (walk_parallel)
  bool recurrent = false;   // some layer has a state that cannot go back
  int streams = 1;
  float embed_scale = 1.f;
  int64_t Wp = 0;       // padded width of the residual stream
  cg_tensor *embed_norm = nullptr, *w_loop = nullptr, *ln_f_bias = nullptr;
  // sequences
  std::vector<uint8_t> open;
  std::vector<int64_t> pos;     // tokens each slot holds
  std::vector<int> cur_slots;   // the current rows
  bool tables_current = false;  // the decode tables describe the current rows
  cg_tensor *tab_run = nullptr, *tab_dec = nullptr;  // row tables of a portion / of decode steps
  int64_t tab_run_words = 0;
  // workspace for `cap` tokens
  int64_t cap = 0, cap_w = 0;
  cg_tensor *x = nullptr, *xn = nullptr, *xcat = nullptr, *y = nullptr, *proj = nullptr, *cv = nullptr, *gl = nullptr, *co = nullptr,
            *ro = nullptr, *att = nullptr, *hact = nullptr, *gu = nullptr, *q = nullptr, *cpk = nullptr, *tok = nullptr, *xw = nullptr,
            *qkv = nullptr, *rn = nullptr, *tinv = nullptr, *kv = nullptr, *lat = nullptr;
  cg_tensor *z = nullptr, *low_gate = nullptr, *u = nullptr, *lru_a = nullptr, *lru_b = nullptr, *y2 = nullptr, *depth = nullptr,
            *side_z = nullptr, *side_h = nullptr, *side_embed = nullptr, *decayed = nullptr;
  int64_t decayed_n = 0;
  int64_t side_p = 0;   // padded width of a layer's token input
  // experts: (token, expert) pairs
  cg_tensor *m_logits = nullptr, *m_ids = nullptr, *m_wts = nullptr, *m_pos = nullptr, *m_tiles = nullptr, *m_xg = nullptr, *m_h = nullptr,
            *m_y = nullptr;
  int64_t m_pairs = 0;
  int64_t tinv_n = 0, kv_n = 0;
  bool keep = false;
  cg_tensor* kept = nullptr;
  int64_t kept_M = 0;

  int act_storage() const { return f32 ? ST_F32 : ST_BF16; }
};

namespace {

int new2(cg_ctx* c, int storage, int64_t a, int64_t b, cg_tensor** out, bool zero = true) {
  drop(*out);
  int64_t d[2] = {a, b};
  CG_TRY(new_tensor(c, CG_F32, storage, d, 2, out));
  if (zero) CG_CUDA(c, cudaMemsetAsync((*out)->data(), 0, (size_t)(a * b) * storage_bytes(storage), c->core->stream));
  return CG_OK;
}

// Rows [r0, r0 + nr) x cols [c0, c0 + nc) of parameter `name` (which must be [rows, cols]) into dst at
// (row, col), in dst's element type.
int place(cg_decoder* D, const std::string& name, int64_t rows, int64_t cols, int64_t r0, int64_t nr, int64_t c0, int64_t nc,
          cg_tensor* dst, int64_t row, int64_t col) {
  cg_ctx* c = D->c;
  cg_tensor* w = nullptr;
  CG_TRY(get_param(D, name, &w));
  if (w->rank != 2 || w->dims[0] != rows || w->dims[1] != cols)
    return fail(c, CG_ERR_SHAPE, "decoder: " + name + " has an unexpected shape");
  Hold h;
  if (dst->storage == ST_BF16) CG_TRY(cg_to_bf16(c, w, &h.t));
  else CG_TRY(as_contiguous_f32(c, w, &h.t));
  const size_t es = storage_bytes(dst->storage);
  CG_CUDA(c, cudaMemcpy2DAsync((char*)dst->data() + (size_t)(row * dst->dims[1] + col) * es, (size_t)dst->dims[1] * es,
                               (const char*)h.t->data() + (size_t)(r0 * cols + c0) * es, (size_t)cols * es, (size_t)nc * es, (size_t)nr,
                               cudaMemcpyDeviceToDevice, c->core->stream));
  return CG_OK;
}
int place_all(cg_decoder* D, const std::string& name, int64_t rows, int64_t cols, cg_tensor* dst, int64_t row, int64_t col = 0) {
  return place(D, name, rows, cols, 0, rows, 0, cols, dst, row, col);
}
// a rank-2 parameter as contiguous f32
int f32_matrix(cg_decoder* D, const std::string& name, int64_t rows, int64_t cols, cg_tensor** out) {
  CG_TRY(new2(D->c, ST_F32, rows, cols, out, false));
  return place_all(D, name, rows, cols, *out, 0);
}

// a vector as it is applied: times a factor, after the 1 a design may add to stored gains
int gains(cg_decoder* D, const std::string& name, int64_t n, cg_tensor** out, float factor = 1.f, bool plus_one = false) {
  if (!plus_one && factor == 1.f) return norm_weight(D, name, n, out);
  Hold w;
  CG_TRY(norm_weight(D, name, n, &w.t));
  CG_TRY(new2(D->c, ST_F32, 1, n, out, false));
  CG_CUDA(D->c, cudaMemcpyAsync((*out)->data(), w.t->data(), (size_t)n * 4, cudaMemcpyDeviceToDevice, D->c->core->stream));
  return k_launch_affine(D->c, (float*)(*out)->data(), n, factor, plus_one ? factor : 0.f);
}
// gains and, of a layer norm, biases
int norm_pair(cg_decoder* D, const std::string& name, cg_tensor** w, cg_tensor** b, float factor = 1.f) {
  CG_TRY(gains(D, name, D->H, w, factor, D->cfg.norm_plus_one != 0));
  return D->cfg.layer_norm ? gains(D, name + ".b", D->H, b, factor) : CG_OK;
}
// n heads of d values each, spread to heads of Dp with zeros between
int head_gains(cg_decoder* D, const std::string& name, int64_t n, int64_t d, int64_t Dp, cg_tensor** out) {
  Hold w;
  CG_TRY(norm_weight(D, name, n * d, &w.t));
  CG_TRY(new2(D->c, ST_F32, n, Dp, out));
  CG_CUDA(D->c, cudaMemcpy2DAsync((*out)->data(), (size_t)Dp * 4, w.t->data(), (size_t)d * 4, (size_t)d * 4, (size_t)n,
                                  cudaMemcpyDeviceToDevice, D->c->core->stream));
  return CG_OK;
}
// the streams' coefficients of a sublayer: all 1 for a plain residual stream
int coefficients(cg_decoder* D, const std::string& name, int64_t n, cg_tensor** out) {
  if (D->cfg.streams > 0) return norm_weight(D, name, n, out);
  CG_TRY(new2(D->c, ST_F32, 1, n, out));
  return k_launch_affine(D->c, (float*)(*out)->data(), n, 1.f, 1.f);
}

// a parameter's values on the host, and the other way round
int download(cg_decoder* D, const std::string& name, int64_t n, std::vector<float>* out) {
  Hold w;
  CG_TRY(norm_weight(D, name, n, &w.t));
  out->resize((size_t)n);
  CG_CUDA(D->c, cudaMemcpyAsync(out->data(), w.t->data(), (size_t)n * 4, cudaMemcpyDeviceToHost, D->c->core->stream));
  CG_CUDA(D->c, cudaStreamSynchronize(D->c->core->stream));
  return CG_OK;
}
int upload(cg_decoder* D, const std::vector<float>& v, cg_tensor** out) {
  CG_TRY(new2(D->c, ST_F32, 1, (int64_t)v.size(), out, false));
  CG_CUDA(D->c, cudaMemcpyAsync((*out)->data(), v.data(), v.size() * 4, cudaMemcpyHostToDevice, D->c->core->stream));
  CG_CUDA(D->c, cudaStreamSynchronize(D->c->core->stream));
  return CG_OK;
}
// entries before and behind a head's distance biases, which kernels may read for keys and rows that do not exist
constexpr int64_t BIAS_PAD = 256;

int rope_tables(cg_decoder* D, const MixedLayer& L, cg_tensor** cos_t, cg_tensor** sin_t) {
  const int64_t half = std::max(L.k.rot_dim / 2, 1);
  CG_TRY(new2(D->c, ST_F32, D->cfg.max_seq, half, cos_t));
  CG_TRY(new2(D->c, ST_F32, D->cfg.max_seq, half, sin_t));
  if (!L.k.rot_dim) return CG_OK;
  PairRope f;
  f.base = L.k.rot_base;
  f.factor = L.k.rot_factor; f.low = L.k.rot_low; f.high = L.k.rot_high; f.original = L.k.rot_original;
  return k_launch_pair_rope_tables(D->c, f, D->cfg.max_seq, L.k.rot_dim, (float*)(*cos_t)->data(), (float*)(*sin_t)->data());
}

// The rows of n heads of d queries or keys at dst's row `row`, Dp rows per head.  Kernels rotate
// neighbouring components; where the design pairs i with i + r / 2, the rows are interleaved, which changes
// neither scores nor norms.
int place_heads(cg_decoder* D, const std::string& name, const cg_layer_config& k, int64_t n, int64_t d, int64_t Dp, cg_tensor* dst,
                int64_t row) {
  const int64_t W = D->H, half = k.rot_half ? k.rot_dim / 2 : 0;
  cg_ctx* c = D->c;
  for (int64_t h = 0; h < n; ++h) CG_TRY(place(D, name, n * d, W, h * d, d, 0, W, dst, row + h * Dp, 0));
  if (half < 2) return CG_OK;
  const size_t es = storage_bytes(dst->storage), line = (size_t)dst->dims[1] * es;
  Hold t;
  CG_TRY(new2(c, dst->storage, 2 * half, dst->dims[1], &t.t, false));
  for (int64_t h = 0; h < n; ++h) {
    char* at = (char*)dst->data() + (size_t)(row + h * Dp) * line;
    CG_CUDA(c, cudaMemcpyAsync(t.t->data(), at, 2 * half * line, cudaMemcpyDeviceToDevice, c->core->stream));
    for (int64_t i = 0; i < 2; ++i)
      CG_CUDA(c, cudaMemcpy2DAsync(at + i * line, 2 * line, (char*)t.t->data() + i * half * line, line, line, (size_t)half,
                                   cudaMemcpyDeviceToDevice, c->core->stream));
  }
  return CG_OK;
}

int finalize_attention(cg_decoder* D, MixedLayer& L, const std::string& mx) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const cg_layer_config& k = L.k;
  const int64_t W = D->H, H = k.heads, G = k.kv_heads, d = k.dim, dv = k.vdim;
  const int st = X.act_storage();
  // head size of the tensor-core kernels; other sizes and f32 only pad to vectors
  const int64_t widest = std::max(d, dv);
  const int Dp = X.f32 ? 0 : widest <= 64 ? 64 : widest <= 128 ? 128 : widest <= 256 ? 256 : 0;
  L.Dk = Dp ? Dp : (int)up8(d);
  L.Dv = L.Do = Dp ? Dp : (int)up8(dv);
  L.gate_off = (int)((H + G) * L.Dk + G * L.Dv);
  L.Np = up8(L.gate_off + (k.gate == 2 ? H * L.Dv : k.gate ? H : 0));
  L.Ko = H * L.Dv;
  CG_TRY(new2(c, st, L.Np, X.Wp, &L.w_in));
  CG_TRY(place_heads(D, mx + "q", k, H, d, L.Dk, L.w_in, 0));
  CG_TRY(place_heads(D, mx + "k", k, G, d, L.Dk, L.w_in, H * L.Dk));
  for (int64_t g = 0; g < G; ++g) CG_TRY(place(D, mx + "v", G * dv, W, g * dv, dv, 0, W, L.w_in, (H + G) * L.Dk + g * L.Dv, 0));
  if (k.gate == 1) CG_TRY(place_all(D, mx + "g", H, W, L.w_in, L.gate_off));
  if (k.gate == 2)
    for (int64_t h = 0; h < H; ++h) CG_TRY(place(D, mx + "g", H * dv, W, h * dv, dv, 0, W, L.w_in, L.gate_off + h * L.Dv, 0));
  if (k.q_temp_every > 0) {
    std::vector<float> t((size_t)D->cfg.max_seq);
    for (size_t p = 0; p < t.size(); ++p) t[p] = (float)(1.0 + k.q_temp_coef * std::log(std::floor((double)(p + 1) / k.q_temp_every) + 1.0));
    CG_TRY(upload(D, t, &L.q_temp));
  }
  if (k.dist_bias) {
    std::vector<float> r1, r2;
    CG_TRY(download(D, mx + "r1", H, &r1));
    CG_TRY(download(D, mx + "r2", H, &r2));
    const int64_t T = D->cfg.max_seq, ld = T + 2 * BIAS_PAD;
    std::vector<float> t((size_t)(H * ld), 0.f);
    for (int64_t h = 0; h < H; ++h)
      for (int64_t x = 0; x < T + BIAS_PAD; ++x) t[(size_t)(h * ld + BIAS_PAD + x)] = (float)((double)r1[h] * std::log1p((double)r2[h] * (double)x));
    CG_TRY(upload(D, t, &L.bias));
  }
  CG_TRY(new2(c, st, X.Wp, L.Ko, &L.w_o));
  for (int64_t h = 0; h < H; ++h) CG_TRY(place(D, mx + "o", W, H * dv, 0, W, h * dv, dv, L.w_o, 0, h * L.Dv));
  if (k.qk_norm == 1) {
    CG_TRY(head_gains(D, mx + "q.norm", H, d, L.Dk, &L.q_gain));
    CG_TRY(head_gains(D, mx + "k.norm", G, d, L.Dk, &L.k_gain));
  }
  if (k.sink) CG_TRY(norm_weight(D, mx + "sink", H, &L.sink));
  return rope_tables(D, L, &L.cos_t, &L.sin_t);
}

// [experts, rows padded to rp, cols padded to cp] from l<i>.mlp.e<j>.<name>
int stack_experts(cg_decoder* D, const std::string& ff, const char* name, int64_t E, int64_t rows, int64_t cols, int64_t rp, int64_t cp,
                  cg_tensor** out) {
  CG_TRY(new2(D->c, D->mixed->act_storage(), E * rp, cp, out));
  for (int64_t e = 0; e < E; ++e) CG_TRY(place_all(D, ff + "e" + std::to_string(e) + "." + name, rows, cols, *out, e * rp));
  return CG_OK;
}

int finalize_experts(cg_decoder* D, MixedLayer& L, const std::string& ff) {
  MixedModel& X = *D->mixed;
  const int64_t W = D->H, F = L.k.ffn, E = L.k.experts;
  CG_TRY(new2(D->c, X.act_storage(), E, X.Wp, &L.router));
  CG_TRY(place_all(D, ff + "router", E, W, L.router, 0));
  if (L.k.correction) CG_TRY(norm_weight(D, ff + "correction", E, &L.correction));
  if (L.k.act != CG_ACT_RELU2) CG_TRY(stack_experts(D, ff, "gate", E, F, W, L.Fp, X.Wp, &L.we_gate));
  CG_TRY(stack_experts(D, ff, "up", E, F, W, L.Fp, X.Wp, &L.we_up));
  return stack_experts(D, ff, "down", E, W, F, X.Wp, L.Fp, &L.we_down);
}

int finalize_latent(cg_decoder* D, MixedLayer& L, const std::string& mx) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const cg_layer_config& k = L.k;
  const int64_t W = D->H, H = k.heads, d = k.dim, r = k.rot_dim, dv = k.vdim, R = k.kv_rank;
  const int st = X.act_storage();
  L.Lw = up16(R + r);
  L.dkv_off = (int)up8(H * (d + r));
  L.Np = up8(L.dkv_off + R + r);
  // head size of the expanded keys and values that the prompt kernels work on
  const int64_t widest = std::max(d + r, dv);
  const int Dp = X.f32 ? 0 : widest <= 64 ? 64 : widest <= 128 ? 128 : widest <= 256 ? 256 : 0;
  L.Dq = Dp ? Dp : (int)(d + r);
  L.Do = Dp ? Dp : (int)dv;
  L.Ko = up8(H * L.Do);
  CG_TRY(new2(c, st, L.Np, X.Wp, &L.w_in));
  CG_TRY(place_all(D, mx + "q", H * (d + r), W, L.w_in, 0));
  CG_TRY(place_all(D, mx + "dkv", R + r, W, L.w_in, L.dkv_off));
  CG_TRY(norm_weight(D, mx + "dkv.norm", R, &L.c_gain));
  CG_TRY(new2(c, st, H * d, R, &L.uk, false));
  CG_TRY(place_all(D, mx + "uk", H * d, R, L.uk, 0));
  CG_TRY(new2(c, st, H * dv, R, &L.uv, false));
  CG_TRY(place_all(D, mx + "uv", H * dv, R, L.uv, 0));
  CG_TRY(new2(c, st, X.Wp, L.Ko, &L.w_o));
  for (int64_t h = 0; h < H; ++h) CG_TRY(place(D, mx + "o", W, H * dv, 0, W, h * dv, dv, L.w_o, 0, h * L.Do));
  if (Dp) {
    // [keys | values] of every head from a cached row in one GEMM: Wuk beside an identity that hands
    // the rotated part through, then Wuv
    CG_TRY(new2(c, ST_BF16, 2 * H * Dp, L.Lw, &L.w_kv));
    std::vector<uint16_t> eye((size_t)(r * L.Lw), 0);
    for (int64_t j = 0; j < r; ++j) eye[(size_t)(j * L.Lw + R + j)] = 0x3F80;  // 1.0
    for (int64_t h = 0; h < H; ++h) {
      CG_TRY(place(D, mx + "uk", H * d, R, h * d, d, 0, R, L.w_kv, h * Dp, 0));
      CG_CUDA(c, cudaMemcpyAsync((uint16_t*)L.w_kv->data() + (h * Dp + d) * L.Lw, eye.data(), eye.size() * 2, cudaMemcpyHostToDevice,
                                 c->core->stream));
      CG_TRY(place(D, mx + "uv", H * dv, R, h * dv, dv, 0, R, L.w_kv, (H + h) * Dp, 0));
    }
    CG_CUDA(c, cudaStreamSynchronize(c->core->stream));
  }
  return rope_tables(D, L, &L.cos_t, &L.sin_t);
}

int finalize_lightning(cg_decoder* D, MixedLayer& L, const std::string& mx) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const cg_layer_config& k = L.k;
  const int64_t W = D->H, H = k.heads, d = k.dim, dv = k.vdim;
  const int st = X.act_storage();
  L.H = L.KH = k.heads;
  L.dk = k.dim; L.dv = k.vdim;
  L.dvs = (int)up8(dv);
  // heads as far apart as the chunk kernels read them, so that the projection itself is their operand
  L.qs = (int)up16(d); L.vs = L.dvs;
  L.q_off = 0; L.k_off = (int)(H * L.qs); L.v_off = 2 * L.k_off;
  L.C = L.v_off + (int)(H * L.vs);
  L.chunked = !X.f32 && chunk_supported(L.dk);
  L.gate_off = L.small_off = L.C;
  L.Np = up8(L.C + H * dv);
  L.Do = L.dv;
  L.Ko = up8(H * dv);
  CG_TRY(new2(c, st, L.Np, X.Wp, &L.w_in));
  for (int64_t h = 0; h < H; ++h) {
    CG_TRY(place(D, mx + "q", H * d, W, h * d, d, 0, W, L.w_in, L.q_off + h * L.qs, 0));
    CG_TRY(place(D, mx + "k", H * d, W, h * d, d, 0, W, L.w_in, L.k_off + h * L.qs, 0));
    CG_TRY(place(D, mx + "v", H * dv, W, h * dv, dv, 0, W, L.w_in, L.v_off + h * L.vs, 0));
  }
  CG_TRY(place_all(D, mx + "g", H * dv, W, L.w_in, L.gate_off));
  CG_TRY(gains(D, mx + "norm", H * dv, &L.norm, L.out_scale()));
  std::vector<float> ld(H);
  for (int64_t h = 0; h < H; ++h) ld[h] = (float)std::log(std::max(L.decay[h], 1e-80));  // (as good as 0 after one token)
  CG_TRY(new2(c, ST_F32, 1, H, &L.log_decay, false));
  CG_CUDA(c, cudaMemcpyAsync(L.log_decay->data(), ld.data(), (size_t)H * 4, cudaMemcpyHostToDevice, c->core->stream));
  CG_CUDA(c, cudaStreamSynchronize(c->core->stream));
  CG_TRY(new2(c, st, X.Wp, L.Ko, &L.w_o));
  return place_all(D, mx + "o", W, H * dv, L.w_o, 0);
}

int finalize_recurrent(cg_decoder* D, MixedLayer& L, const std::string& mx) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const cg_layer_config& k = L.k;
  const int64_t W = D->H, taps = k.conv;
  const bool delta = k.mixer == CG_MIX_DELTA;
  const int st = X.act_storage();
  L.H = k.heads;
  L.dv = k.vdim;
  L.dvs = (int)up8(L.dv);
  const int64_t inner = (int64_t)L.H * L.dv;
  L.KH = delta ? k.kv_heads : k.groups;
  L.dk = delta ? k.dim : k.state;
  const int64_t kk = (int64_t)L.KH * L.dk;
  L.C = (int)(inner + 2 * kk);
  L.chunked = !X.f32 && chunk_supported(L.dk);
  L.qs = L.dk; L.vs = L.dv;
  L.gate_off = (int)up8(L.C);
  L.small_off = (int)up8(L.gate_off + inner);
  L.Np = up8(L.small_off + (delta ? 2 : 1) * L.H);
  CG_TRY(new2(c, st, L.Np, X.Wp, &L.w_in));
  CG_TRY(new2(c, ST_F32, L.C, taps, &L.conv_w, false));
  if (delta) {
    L.q_off = 0; L.k_off = (int)kk; L.v_off = (int)(2 * kk);
    CG_TRY(place_all(D, mx + "q", kk, W, L.w_in, L.q_off));
    CG_TRY(place_all(D, mx + "k", kk, W, L.w_in, L.k_off));
    CG_TRY(place_all(D, mx + "v", inner, W, L.w_in, L.v_off));
    CG_TRY(place_all(D, mx + "g", inner, W, L.w_in, L.gate_off));
    CG_TRY(place_all(D, mx + "b", L.H, W, L.w_in, L.small_off));
    CG_TRY(place_all(D, mx + "a", L.H, W, L.w_in, L.small_off + L.H));
    CG_TRY(place_all(D, mx + "q.conv", kk, taps, L.conv_w, L.q_off));
    CG_TRY(place_all(D, mx + "k.conv", kk, taps, L.conv_w, L.k_off));
    CG_TRY(place_all(D, mx + "v.conv", inner, taps, L.conv_w, L.v_off));
    CG_TRY(gains(D, mx + "norm", L.dv, &L.norm, L.out_scale()));
  } else {
    // stored [z | x | B | C | dt]; the convolved channels come first here
    L.v_off = 0; L.k_off = (int)inner; L.q_off = (int)(inner + kk);
    const int64_t rows = 2 * inner + 2 * kk + L.H;
    CG_TRY(place(D, mx + "in", rows, W, inner, L.C, 0, W, L.w_in, 0, 0));
    CG_TRY(place(D, mx + "in", rows, W, 0, inner, 0, W, L.w_in, L.gate_off, 0));
    CG_TRY(place(D, mx + "in", rows, W, inner + L.C, L.H, 0, W, L.w_in, L.small_off, 0));
    CG_TRY(place_all(D, mx + "conv", L.C, taps, L.conv_w, 0));
    CG_TRY(norm_weight(D, mx + "conv.b", L.C, &L.conv_b));
    CG_TRY(norm_weight(D, mx + "D", L.H, &L.dskip));
    CG_TRY(gains(D, mx + "norm", inner, &L.norm, L.out_scale()));
  }
  CG_TRY(norm_weight(D, mx + "A_log", L.H, &L.a_log));
  CG_TRY(norm_weight(D, mx + "dt_bias", L.H, &L.dt_bias));
  L.Do = L.dv;
  L.Ko = up8(inner);
  CG_TRY(new2(c, st, X.Wp, L.Ko, &L.w_o));
  return place_all(D, mx + "o", W, inner, L.w_o, 0);
}

// rows of the first factor of a low-rank projection, as many as its tensor has
int low_rank_of(cg_decoder* D, const std::string& name, int* rank) {
  cg_tensor* w = nullptr;
  CG_TRY(get_param(D, name, &w));
  if (w->rank != 2 || w->dims[0] < 1 || w->dims[0] > 4096) return fail(D->c, CG_ERR_SHAPE, "decoder: " + name + " has an unexpected shape");
  *rank = (int)w->dims[0];
  return CG_OK;
}

// Decays per key channel: z = W_a2 (W_a1 h), its heads zs columns apart, ln g = -coef softplus(sign (z + bias)).
int finalize_key_decay(cg_decoder* D, MixedLayer& L, const std::string& mx) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const cg_layer_config& k = L.k;
  const bool delta = L.delta();
  const int64_t W = D->H, H = k.heads, KH = delta ? k.kv_heads : H, d = k.dim, dv = k.vdim;
  const int st = X.act_storage();
  L.H = (int)H; L.KH = (int)KH;
  L.dk = k.dim; L.dv = k.vdim;
  L.dvs = (int)up8(dv);
  L.zs = (int)up16(d);
  // without convolutions the projection itself is the chunk kernels' operand: heads as far apart as they read them
  L.qs = delta ? L.dk : L.zs;
  L.vs = delta ? L.dv : L.dvs;
  L.q_off = 0; L.k_off = (int)(KH * L.qs); L.v_off = 2 * L.k_off;
  L.C = L.v_off + (int)(H * L.vs);
  L.chunked = !X.f32 && chunk_supported(L.dk);
  int ra = 0, rg = 0;
  CG_TRY(low_rank_of(D, mx + "a1", &ra));
  if (delta) CG_TRY(low_rank_of(D, mx + "g1", &rg));
  L.a_rank = (int)up8(ra); L.g_rank = (int)up8(rg);
  L.gate_off = (int)up8(L.C);
  L.a1_off = (int)up8(L.gate_off + (delta ? 0 : H * dv));
  L.g1_off = L.a1_off + L.a_rank;
  L.small_off = L.g1_off + L.g_rank;
  L.Np = up8(L.small_off + (delta ? H : 0));
  CG_TRY(new2(c, st, L.Np, X.Wp, &L.w_in));
  for (int64_t h = 0; h < KH; ++h) {
    CG_TRY(place(D, mx + "q", KH * d, W, h * d, d, 0, W, L.w_in, L.q_off + h * L.qs, 0));
    CG_TRY(place(D, mx + "k", KH * d, W, h * d, d, 0, W, L.w_in, L.k_off + h * L.qs, 0));
  }
  for (int64_t h = 0; h < H; ++h) CG_TRY(place(D, mx + "v", H * dv, W, h * dv, dv, 0, W, L.w_in, L.v_off + h * L.vs, 0));
  CG_TRY(place_all(D, mx + "a1", ra, W, L.w_in, L.a1_off));
  CG_TRY(new2(c, st, H * L.zs, L.a_rank, &L.w_a2));
  for (int64_t h = 0; h < H; ++h) CG_TRY(place(D, mx + "a2", H * d, ra, h * d, d, 0, ra, L.w_a2, h * L.zs, 0));
  CG_TRY(head_gains(D, mx + (delta ? "dt_bias" : "a2.b"), H, d, L.zs, &L.dt_bias));
  CG_TRY(gains(D, mx + "norm", dv, &L.norm, L.out_scale()));
  std::vector<float> f((size_t)H, (float)(1.0 / k.tau));
  if (delta) {
    CG_TRY(download(D, mx + "A_log", H, &f));
    for (float& x : f) x = (float)std::exp((double)x);
    CG_TRY(place_all(D, mx + "b", H, W, L.w_in, L.small_off));
    CG_TRY(place_all(D, mx + "g1", rg, W, L.w_in, L.g1_off));
    CG_TRY(new2(c, st, H * dv, L.g_rank, &L.w_g2));
    CG_TRY(place_all(D, mx + "g2", H * dv, rg, L.w_g2, 0));
    CG_TRY(new2(c, ST_F32, L.C, k.conv, &L.conv_w, false));
    CG_TRY(place_all(D, mx + "q.conv", KH * d, k.conv, L.conv_w, L.q_off));
    CG_TRY(place_all(D, mx + "k.conv", KH * d, k.conv, L.conv_w, L.k_off));
    CG_TRY(place_all(D, mx + "v.conv", H * dv, k.conv, L.conv_w, L.v_off));
  } else {
    CG_TRY(place_all(D, mx + "g", H * dv, W, L.w_in, L.gate_off));
  }
  CG_TRY(upload(D, f, &L.coef));
  L.Do = L.dv;
  L.Ko = up8(H * dv);
  CG_TRY(new2(c, st, X.Wp, L.Ko, &L.w_o));
  return place_all(D, mx + "o", W, H * dv, L.w_o, 0);
}

// [blocks, n, n] as [blocks n, n] in the activations' type
int block_diagonal(cg_decoder* D, const std::string& name, int64_t blocks, int64_t n, cg_tensor** out) {
  cg_ctx* c = D->c;
  cg_tensor* w = nullptr;
  CG_TRY(get_param(D, name, &w));
  if (w->rank != 3 || w->dims[0] != blocks || w->dims[1] != n || w->dims[2] != n)
    return fail(c, CG_ERR_SHAPE, "decoder: " + name + " has an unexpected shape");
  Hold h;
  const int st = D->mixed->act_storage();
  if (st == ST_BF16) CG_TRY(cg_to_bf16(c, w, &h.t));
  else CG_TRY(as_contiguous_f32(c, w, &h.t));
  CG_TRY(new2(c, st, blocks * n, n, out, false));
  CG_CUDA(c, cudaMemcpyAsync((*out)->data(), h.t->data(), (size_t)(blocks * n * n) * storage_bytes(st), cudaMemcpyDeviceToDevice, c->core->stream));
  return CG_OK;
}

int finalize_lru(cg_decoder* D, MixedLayer& L, const std::string& mx) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int64_t W = D->H, B = L.k.heads, n = L.k.vdim, C = B * n;
  const int st = X.act_storage();
  L.C = (int)C;
  L.H = (int)B; L.dv = L.dvs = (int)n;
  L.x_off = (int)up8(C);
  L.Np = up8(L.x_off + C);
  L.Ko = up8(C);
  L.Do = (int)n;
  CG_TRY(new2(c, st, L.Np, X.Wp, &L.w_in));
  CG_TRY(place_all(D, mx + "y", C, W, L.w_in, 0));
  CG_TRY(place_all(D, mx + "x", C, W, L.w_in, L.x_off));
  CG_TRY(gains(D, mx + "y.b", C, &L.yb));
  CG_TRY(gains(D, mx + "x.b", C, &L.xb));
  CG_TRY(f32_matrix(D, mx + "conv", C, L.k.conv, &L.conv_w));
  CG_TRY(gains(D, mx + "conv.b", C, &L.conv_b));
  CG_TRY(block_diagonal(D, mx + "ra", B, n, &L.ra));
  CG_TRY(block_diagonal(D, mx + "ri", B, n, &L.ri));
  CG_TRY(gains(D, mx + "ra.b", C, &L.ra_b));
  CG_TRY(gains(D, mx + "ri.b", C, &L.ri_b));
  std::vector<float> f;
  CG_TRY(download(D, mx + "lam", C, &f));
  for (float& x : f) x = (float)(-8.0 * (std::max((double)x, 0.0) + std::log1p(std::exp(-std::fabs((double)x)))));
  CG_TRY(upload(D, f, &L.coef));
  CG_TRY(new2(c, st, X.Wp, L.Ko, &L.w_o));
  return place_all(D, mx + "o", W, C, L.w_o, 0);
}

int finalize_mixer(cg_decoder* D, MixedLayer& L, const std::string& mx) {
  switch (L.k.mixer) {
    case CG_MIX_ATTENTION: return finalize_attention(D, L, mx);
    case CG_MIX_LATENT: return finalize_latent(D, L, mx);
    case CG_MIX_LIGHTNING: return finalize_lightning(D, L, mx);
    case CG_MIX_CHANNEL_DELTA:
    case CG_MIX_GLA: return finalize_key_decay(D, L, mx);
    case CG_MIX_LRU: return finalize_lru(D, L, mx);
    default: return finalize_recurrent(D, L, mx);
  }
}

// two mixers' projections become one matrix, and their output projections one whose rows span both (unless each
// result has a norm of its own)
int finalize_beside(cg_decoder* D, MixedLayer& L, const std::string& mx) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  MixedLayer& R = *L.beside;
  CG_TRY(finalize_mixer(D, L, mx + "left."));
  CG_TRY(finalize_mixer(D, R, mx + "right."));
  R.in_row = L.Np;
  R.out_col = L.Ko;
  Hold in, out;
  CG_TRY(new2(c, X.act_storage(), L.in_width(), X.Wp, &in.t));
  if (!L.k.out_norm) CG_TRY(new2(c, X.act_storage(), X.Wp, L.out_width(), &out.t));
  const size_t es = storage_bytes(X.act_storage());
  for (MixedLayer* m : {&L, &R}) {
    CG_CUDA(c, cudaMemcpyAsync((char*)in.t->data() + (size_t)(m->in_row * X.Wp) * es, m->w_in->data(), (size_t)(m->Np * X.Wp) * es,
                               cudaMemcpyDeviceToDevice, c->core->stream));
    if (!L.k.out_norm) CG_CUDA(c, cudaMemcpy2DAsync((char*)out.t->data() + (size_t)m->out_col * es, (size_t)L.out_width() * es, m->w_o->data(), (size_t)m->Ko * es,
                                 (size_t)m->Ko * es, (size_t)X.Wp, cudaMemcpyDeviceToDevice, c->core->stream));
    drop(m->w_in);
    if (!L.k.out_norm) drop(m->w_o);
  }
  L.w_in = in.take();
  if (!L.k.out_norm) L.w_o = out.take();
  R.w_in = L.w_in;
  R.w_in->rc++;
  if (L.k.out_norm) {
    CG_TRY(gains(D, mx + "left.out", D->H, &L.out_gain, 0.5f));
    CG_TRY(gains(D, mx + "right.out", D->H, &R.out_gain, 0.5f));
  }
  return CG_OK;
}

void forget_graph(cg_decoder* D) {
  if (D->graph) { cudaGraphExecDestroy(D->graph); D->graph = nullptr; }
}

int ensure_mixed(cg_decoder* D, int64_t M) {
  MixedModel& X = *D->mixed;
  if (M <= X.cap) return CG_OK;
  cg_ctx* c = D->c;
  forget_graph(D);  // it holds the old buffers
  int64_t np = 0, cc = 0, hh = 0, inner = 0, ko = 0, fp = 0, qw = 0, lw = 0, qkv = 0, kh = 0, top = 0, experts = 0, fe = 0;
  int64_t zw = 0, gw = 0, lru = 0;
  auto count_mixer = [&](const MixedLayer& L) {
    if (L.k.mixer == CG_MIX_ATTENTION) {
      qw = std::max<int64_t>(qw, (int64_t)L.k.heads * L.Dk);
    } else if (L.k.mixer == CG_MIX_LATENT) {
      qw = std::max<int64_t>(qw, (int64_t)L.k.heads * L.Dq);
      lw = std::max(lw, L.Lw);
    } else if (L.lru()) {
      lru = std::max<int64_t>(lru, L.C);
    } else {
      if (L.key_decay()) {
        zw = std::max<int64_t>(zw, (int64_t)L.H * L.zs);
        if (L.w_g2) gw = std::max<int64_t>(gw, (int64_t)L.H * L.dv);
      }
      cc = std::max<int64_t>(cc, up8(L.C));
      hh = std::max<int64_t>(hh, L.H);
      inner = std::max<int64_t>(inner, (int64_t)L.H * L.dvs);
      if (L.chunked) {
        qkv = std::max<int64_t>(qkv, 2 * L.KH * up16(L.dk) + (int64_t)L.H * L.dvs);
        kh = std::max<int64_t>(kh, L.KH);
      }
    }
  };
  for (const MixedLayer& L : X.layers) {
    if (!L.w_in) continue;  // another layer's parameters
    np = std::max(np, L.in_width());
    ko = std::max(ko, L.out_width());
    fp = std::max(fp, L.Fd);
    if (L.k.experts) {
      top = std::max<int64_t>(top, L.k.top_k);
      experts = std::max<int64_t>(experts, L.k.experts);
      fe = std::max(fe, L.Fp);
    }
    count_mixer(L);
    if (L.beside) count_mixer(*L.beside);
  }
  const int st = X.act_storage();
  CG_TRY(new2(c, ST_F32, M * X.streams, X.Wp, &X.x));
  CG_TRY(new2(c, st, M, X.Wp, &X.xn));
  CG_TRY(new2(c, ST_F32, M, X.Wp, &X.y));
  if (X.loop) CG_TRY(new2(c, st, M, 2 * X.Wp, &X.xcat));
  if (X.parallel) {
    CG_TRY(new2(c, ST_F32, 2 * M, X.Wp, &X.y2));
    if (D->cfg.depth_average) CG_TRY(new2(c, ST_F32, (int64_t)(X.layers.size() + 1) * M, X.Wp, &X.depth));
    if (X.side_p) {
      CG_TRY(new2(c, ST_F32, M, X.side_p, &X.side_z));
      CG_TRY(new2(c, st, M, X.side_p, &X.side_h));
    }
  }
  if (zw) CG_TRY(new2(c, ST_F32, M, zw, &X.z));
  if (gw) CG_TRY(new2(c, ST_F32, M, gw, &X.low_gate));
  if (lru) {
    CG_TRY(new2(c, st, M, lru, &X.u));
    CG_TRY(new2(c, ST_F32, M, lru, &X.lru_a));
    CG_TRY(new2(c, ST_F32, M, lru, &X.lru_b));
  }
  CG_TRY(new2(c, ST_F32, M, np, &X.proj));
  CG_TRY(new2(c, st, M, ko, &X.att));
  if (fp) {
    CG_TRY(new2(c, st, M, fp, &X.hact));
    if (X.f32) CG_TRY(new2(c, ST_F32, M, 2 * fp, &X.gu));
  }
  if (cc) {
    CG_TRY(new2(c, ST_F32, M, cc, &X.cv));
    CG_TRY(new2(c, ST_F32, M, hh, &X.gl));
    CG_TRY(new2(c, ST_F32, M, hh, &X.co));
    CG_TRY(new2(c, ST_F32, M, inner, &X.ro));
  }
  if (qkv) {
    CG_TRY(new2(c, ST_BF16, M, qkv, &X.qkv));
    CG_TRY(new2(c, ST_F32, 2 * M, kh, &X.rn));
  }
  if (!X.f32) {
    size_t lat = 0;
    for (const MixedLayer& L : X.layers)
      if (L.k.mixer == CG_MIX_LATENT) {
        LatentArgs a;
        a.H = L.k.heads; a.R = L.k.kv_rank; a.Lw = L.Lw;
        lat = std::max(lat, latent_decode_scratch(a, std::min<int64_t>(M, LATENT_DECODE_TOKENS)));
      }
    if (lat) CG_TRY(new2(c, ST_F32, (int64_t)(lat + 3) / 4, 1, &X.lat));
  }
  if (qw) {
    CG_TRY(new2(c, st, M, qw, &X.q));
    if (lw) CG_TRY(new2(c, st, M, lw, &X.cpk));
  }
  if (top) {
    const int64_t P = M * top;
    CG_TRY(new2(c, ST_F32, M, experts, &X.m_logits));
    CG_TRY(new2(c, ST_U32, P, 1, &X.m_ids));
    CG_TRY(new2(c, ST_F32, P, 1, &X.m_wts));
    CG_TRY(new2(c, ST_U32, P, 1, &X.m_pos));
    CG_TRY(new2(c, ST_U32, 3 * P + 4, 1, &X.m_tiles));
    CG_TRY(new2(c, st, P, X.Wp, &X.m_xg));
    CG_TRY(new2(c, st, P, fe, &X.m_h));
    CG_TRY(new2(c, ST_F32, P, X.Wp, &X.m_y));
    X.m_pairs = P;
  }
  drop(X.tok);
  CG_TRY(new_tensor(c, CG_U32, ST_U32, &M, 1, &X.tok));
  X.cap = M;
  return CG_OK;
}

// out[M, N] = x[M, K] w[row0 .. row0 + N, K]^T; out_mode (of the GEMMs) 0 f32 or, only in a bf16 context,
// 1 bf16, 4 bf16 of the square of relu, 6 bf16 of gelu(product + bias)
int lin(cg_decoder* D, const void* x, int64_t ldx, int64_t M, const cg_tensor* w, int64_t row0, int64_t N, void* out, int64_t ldo,
        int out_mode = 0, const float* bias = nullptr) {
  cg_ctx* c = D->c;
  const int64_t K = w->dims[1];
  if (D->mixed->f32)
    return gemm_nt_f32(c, (const float*)x, ldx, (const float*)w->data() + row0 * K, K, (float*)out, ldo, M, N, K);
  const __nv_bfloat16* xb = (const __nv_bfloat16*)x;
  const __nv_bfloat16* wb = (const __nv_bfloat16*)w->data() + row0 * K;
  if (gemm_dec_supported(M, K)) {
    DecGemm g;
    g.x = xb; g.ldx = ldx; g.w = wb; g.ldw = K; g.w_rows = N;
    g.out = out; g.ldo = ldo; g.residual = bias; g.out_mode = out_mode;
    g.push = nullptr; g.dual = 0; g.act = 0;
    g.M = M; g.N = N; g.K = K;
    return gemm_dec(c, g);
  }
  const int splits = gemm_tc_pick_splits(M, N, K);
  float* ws = (int64_t)splits * M * N <= D->splitk_floats ? (float*)D->splitk->data() : nullptr;
  return gemm_tc(c, xb, ldx, wb, K, out, ldo, bias, M, N, K, out_mode, splits, ws);
}

// Rows of a matrix some columns wide: where the first starts, and from one to the next.
struct Rows {
  void* p = nullptr;
  int64_t ld = 0;
};

// hact = act(x gate^T) * (x up^T)
int glu(cg_decoder* D, const MixedLayer& L, const void* x, int64_t M) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int64_t K = X.Wp, F = L.Fd;
  if (X.f32) {
    CG_TRY(lin(D, x, K, M, L.w_gu, 0, 2 * F, X.gu->data(), 2 * F));
    return k_launch_glu_f32(c, (const float*)X.gu->data(), M, F, L.k.act, (float*)X.hact->data());
  }
  const __nv_bfloat16* xb = (const __nv_bfloat16*)x;
  const __nv_bfloat16* w = (const __nv_bfloat16*)L.w_gu->data();
  if (gemm_dec_supported(M, K)) {
    DecGemm g;
    g.x = xb; g.ldx = K; g.w = w; g.ldw = K; g.w_rows = 2 * F;
    g.out = X.hact->data(); g.ldo = F; g.residual = nullptr; g.out_mode = 1;
    g.push = nullptr; g.dual = 1; g.act = L.k.act;
    g.M = M; g.N = F; g.K = K;
    return gemm_dec(c, g);
  }
  return gemm_tc_pair(c, xb, K, w, K, (__nv_bfloat16*)X.hact->data(), F, M, F, K, L.k.act);
}

// units = gelu(up h + b) of the rows h = xn
int gelu_units(cg_decoder* D, const MixedLayer& L, int64_t M, Rows units) {
  MixedModel& X = *D->mixed;
  const float* bias = (const float*)L.up_bias->data();
  CG_TRY(lin(D, X.xn->data(), X.Wp, M, L.w_gu, 0, L.Fd, units.p, units.ld, X.f32 ? 0 : 6, bias));
  if (!X.f32) return CG_OK;
  return k_launch_bias_gelu_f32(D->c, (const float*)units.p, units.ld, bias, M, L.Fd, (float*)units.p, units.ld);
}

// y = the dense feed-forward or the shared expert of the rows xn, without the last bias
int dense_ff(cg_decoder* D, const MixedLayer& L, int64_t M) {
  MixedModel& X = *D->mixed;
  if (L.k.act == CG_ACT_GELU1) {
    CG_TRY(gelu_units(D, L, M, Rows{X.hact->data(), L.Fd}));
  } else if (L.k.act == CG_ACT_RELU2) {
    CG_TRY(lin(D, X.xn->data(), X.Wp, M, L.w_gu, 0, L.Fd, X.hact->data(), L.Fd, X.f32 ? 0 : 4));
    if (X.f32) CG_TRY(k_launch_relu2_f32(D->c, (float*)X.hact->data(), M * L.Fd));
  } else {
    CG_TRY(glu(D, L, X.xn->data(), M));
  }
  return lin(D, X.hact->data(), L.Fd, M, L.w_down, 0, X.Wp, X.y->data(), X.Wp);
}

// m_y[m_pos[pair]] = the chosen experts' results for the rows xn, m_wts their weights (on the rows x itself
// where the weights go onto the inputs)
int experts_ff(cg_decoder* D, const MixedLayer& L, int64_t M) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  MoeArgs a;
  a.H = (int)X.Wp; a.E = a.El = L.k.experts; a.e_lo = 0; a.k = L.k.top_k; a.Fe = (int)L.Fp;
  a.norm_topk = 0; a.act = L.k.act; a.act_limit = (float)L.k.act_limit;
  a.correction = L.correction ? (const float*)L.correction->data() : nullptr;
  a.router_scale = (float)L.k.router_scale;
  a.sigmoid = L.k.scoring; a.weigh_input = L.k.weigh_input;
  a.x = (const float*)X.x->data();
  a.M = M;
  a.logits = (float*)X.m_logits->data();
  a.w.ids = (uint32_t*)X.m_ids->data();
  a.w.wts = (float*)X.m_wts->data();
  a.w.pos = (int32_t*)X.m_pos->data();
  int32_t* t = (int32_t*)X.m_tiles->data();
  a.w.tile_expert = t; a.w.tile_row0 = t + X.m_pairs; a.w.tile_rows = t + 2 * X.m_pairs; a.w.n_tiles = t + 3 * X.m_pairs;
  a.w.xg = (__nv_bfloat16*)X.m_xg->data();
  a.w.h = (__nv_bfloat16*)X.m_h->data();
  a.w.y = (float*)X.m_y->data();
  CG_TRY(lin(D, X.xn->data(), X.Wp, M, L.router, 0, a.E, a.logits, a.E));
  CG_TRY(moe_topk(c, a));
  if (X.f32)
    return moe_experts_f32(c, a, (const float*)X.xn->data(), L.we_gate ? (const float*)L.we_gate->data() : nullptr, (const float*)L.we_up->data(),
                           (const float*)L.we_down->data(), (float*)X.m_h->data());
  a.xn = (__nv_bfloat16*)X.xn->data();
  a.w_gate = L.we_gate ? (const __nv_bfloat16*)L.we_gate->data() : nullptr;
  a.w_up = (const __nv_bfloat16*)L.we_up->data();
  a.w_down = (const __nv_bfloat16*)L.we_down->data();
  return moe_experts(c, a);
}

// What the host knows about a portion: per row its new tokens and the position of the first.
struct Portion {
  std::vector<int> slots, lens;
  std::vector<int64_t> pos0;
  int64_t M = 0;
  int max_len = 0;
};

// words of the row tables: slot, start, pos0, tok_row and, for chunks of RECUR_CHUNK tokens, the first
// chunk of every row, the chunks' first tokens and their lengths
int64_t table_words(int64_t rows, int64_t M) {
  return rows + (rows + 1) + rows + M + (rows + 1) + 2 * (M / RECUR_CHUNK + rows);
}
struct Chunks {
  const int32_t *tok, *len, *row_chunk;
  int n;
};

int write_tables(cg_decoder* D, const Portion& p, cg_tensor* dst, RowsDev* rd, Chunks* ch) {
  cg_ctx* c = D->c;
  const int R = (int)p.slots.size();
  std::vector<int32_t> t((size_t)table_words(R, p.M));
  int32_t *slot = t.data(), *start = slot + R, *pos0 = start + R + 1, *tr = pos0 + R;
  int32_t at = 0;
  for (int r = 0; r < R; ++r) {
    slot[r] = p.slots[r];
    start[r] = at;
    pos0[r] = (int32_t)p.pos0[r];
    for (int i = 0; i < p.lens[r]; ++i) tr[at++] = r;
  }
  start[R] = at;
  int32_t *rc = tr + p.M, *ct = rc + R + 1;
  std::vector<int32_t> lens;
  int nc = 0;
  for (int r = 0; r < R; ++r) {
    rc[r] = nc;
    for (int i = 0; i < p.lens[r]; i += RECUR_CHUNK) {
      ct[nc++] = start[r] + i;
      lens.push_back(std::min(RECUR_CHUNK, p.lens[r] - i));
    }
  }
  rc[R] = nc;
  std::copy(lens.begin(), lens.end(), ct + nc);
  CG_CUDA(c, cudaMemcpyAsync(dst->data(), t.data(), t.size() * 4, cudaMemcpyHostToDevice, c->core->stream));
  const int32_t* d = (const int32_t*)dst->data();
  rd->slot = d; rd->start = d + R; rd->pos0 = d + 2 * R + 1; rd->tok_row = d + 3 * R + 1;
  rd->step = D->pos_dev();
  rd->rows = R;
  rd->M = p.M;
  ch->row_chunk = rd->tok_row + p.M;
  ch->tok = ch->row_chunk + R + 1;
  ch->len = ch->tok + nc;
  ch->n = nc;
  return CG_OK;
}

// A buffer that prompts of a new length may have to grow (never part of a captured graph).
int grow(cg_ctx* c, int storage, int64_t n, cg_tensor** t, int64_t* have) {
  if (n <= *have) return CG_OK;
  CG_TRY(new2(c, storage, n, 1, t, false));
  *have = n;
  return CG_OK;
}

// One token per row: norms, rotation, cache append and attention in one kernel.  Longer rows: a pass
// that norms, rotates and appends, then the prompt attention on the tensor cores.  f32, and sizes those
// kernels do not have: one block per token and head.
int attention_layer(cg_decoder* D, const MixedLayer& L, MixedRun& run, const RowsDev& rd, const Portion* p, Rows in, Rows out) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const cg_layer_config& k = L.k;
  const float* proj = (const float*)in.p;
  const float* gate = k.gate ? proj + L.gate_off : nullptr;
  const float* q_gain = L.q_gain ? (const float*)L.q_gain->data() : nullptr;
  const float* k_gain = L.k_gain ? (const float*)L.k_gain->data() : nullptr;
  const float* sink = L.sink ? (const float*)L.sink->data() : nullptr;
  const float* q_temp = L.q_temp ? (const float*)L.q_temp->data() : nullptr;
  const float* bias = L.bias ? (const float*)L.bias->data() + BIAS_PAD : nullptr;
  const int64_t ld_bias = D->cfg.max_seq + 2 * BIAS_PAD;
  const bool tensor = !X.f32 && L.Dk == L.Dv && (L.Dk == 64 || L.Dk == 128 || L.Dk == 256);
  if (tensor && (!p || p->max_len == 1) && k.heads / k.kv_heads <= 8) {
    AttnDecArgs f{};
    f.qkv = proj; f.ld_qkv = in.ld;
    f.cos_t = (const float*)L.cos_t->data(); f.sin_t = (const float*)L.sin_t->data();
    f.q_gamma = q_gain; f.k_gamma = k_gain; f.norm_eps = D->cfg.rms_eps;
    f.k_cache = (__nv_bfloat16*)run.cache->data(); f.v_cache = (__nv_bfloat16*)run.cache_v->data();
    f.out = (__nv_bfloat16*)out.p; f.ld_out = out.ld;
    f.head_norm = k.qk_norm == 2; f.keep_first = k.keep_first;
    f.gate = gate; f.ld_gate = in.ld; f.out_scale = L.out_scale();
    f.Tmax = D->cfg.max_seq; f.B = rd.rows;
    f.nh = k.heads; f.nkv = k.kv_heads; f.d = L.Dk;
    f.window = k.window; f.rows = rd; f.rot_dims = k.rot_dim; f.norm_dim = k.dim;
    f.scale = (float)k.scale; f.sink = sink;
    f.wide_gate = k.gate == 2; f.q_temp = q_temp; f.bias = bias; f.ld_bias = ld_bias;
    const int64_t reach = k.window > 0 ? std::min<int64_t>((int64_t)k.window + k.keep_first, f.Tmax) : f.Tmax;
    f.splits = attn_dec_splits(reach, f.B * f.nkv, f.d);
    return k_launch_attn_dec(c, f);
  }
  RowsAttnArgs a;
  a.proj = proj; a.ldp = in.ld;
  a.H = k.heads; a.G = k.kv_heads; a.d = k.dim; a.dv = k.vdim; a.Dk = L.Dk; a.Dv = L.Dv;
  a.q_gain = q_gain; a.k_gain = k_gain; a.eps = D->cfg.rms_eps; a.scale = (float)k.scale;
  a.rot = k.rot_dim;
  a.cos_t = (const float*)L.cos_t->data(); a.sin_t = (const float*)L.sin_t->data();
  a.window = k.window; a.keep_first = k.keep_first; a.sink = sink;
  a.head_norm = k.qk_norm == 2;
  a.gate = gate; a.out_scale = L.out_scale();
  a.wide_gate = k.gate == 2; a.q_temp = q_temp; a.bias = bias; a.ld_bias = ld_bias;
  a.q = X.q->data(); a.k_cache = run.cache->data(); a.v_cache = run.cache_v->data();
  a.Tmax = D->cfg.max_seq; a.slots = D->cfg.max_batch;
  a.att = out.p; a.ld_att = out.ld;
  a.bf16 = X.f32 ? 0 : 1;
  a.rows = rd;
  CG_TRY(k_launch_rows_qkv(c, a));
  if (!tensor || !p) return k_launch_rows_attn(c, a);
  AttnArgs t{};
  t.q = (const __nv_bfloat16*)a.q;
  t.k_cache = (const __nv_bfloat16*)a.k_cache; t.v_cache = (const __nv_bfloat16*)a.v_cache;
  t.out = (__nv_bfloat16*)a.att;
  t.B = a.slots; t.S = p->max_len; t.Tmax = a.Tmax;
  t.nh = a.H; t.nkv = a.G; t.d = L.Dk;
  t.window = a.window; t.keep_first = a.keep_first; t.scale = a.scale; t.sink = sink; t.rows = rd;
  t.wide_gate = a.wide_gate; t.bias = bias; t.ld_bias = ld_bias;
  t.gate = gate; t.ld_gate = in.ld; t.out_scale = a.out_scale; t.ld_out = out.ld;
  return k_launch_attn_prefill(c, t);
}

// A few new tokens: attention in the cached rows' space.  Prompts: the cached rows are expanded to
// keys and values of Dq values per head, token after token, and run through the prompt attention.
// f32, and sizes those kernels do not have: one block per token and head.
int latent_layer(cg_decoder* D, const MixedLayer& L, MixedRun& run, const RowsDev& rd, const Portion* p) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  CG_TRY(lin(D, X.xn->data(), X.Wp, rd.M, L.w_in, 0, L.Np, X.proj->data(), L.Np));
  LatentArgs a;
  a.proj = (const float*)X.proj->data(); a.ldp = L.Np; a.dkv_off = L.dkv_off;
  a.H = L.k.heads; a.d = L.k.dim; a.r = L.k.rot_dim; a.dv = L.k.vdim; a.R = L.k.kv_rank;
  a.scale = (float)L.k.scale; a.eps = D->cfg.rms_eps;
  a.cos_t = (const float*)L.cos_t->data(); a.sin_t = (const float*)L.sin_t->data();
  a.c_gain = (const float*)L.c_gain->data();
  a.cache = run.cache->data(); a.Lw = L.Lw; a.Tmax = D->cfg.max_seq;
  a.q_out = X.q->data(); a.Dq = L.Dq;
  a.c_out = nullptr;
  a.uk = L.uk->data(); a.uv = L.uv->data();
  a.att = X.att->data(); a.ld_att = L.Ko; a.Do = L.Do;
  a.bf16 = X.f32 ? 0 : 1;
  a.rows = rd;
  if (!X.f32 && (!p || p->max_len <= 4) && rd.M <= LATENT_DECODE_TOKENS && latent_decode_supported(a.d, a.R, a.Lw))
    return k_launch_latent_decode(c, a, X.lat->data());
  if (!L.w_kv || !p) {
    CG_TRY(k_launch_latent_prep(c, a));
    return k_launch_latent_attn(c, a);
  }
  const int R = rd.rows;
  const int64_t Dp = L.Dq, kvw = 2 * a.H * Dp, es = 2;
  bool equal = true, fresh = true;
  int64_t ctx = 0;
  for (int r = 0; r < R; ++r) {
    equal = equal && p->lens[r] == p->lens[0] && p->pos0[r] == p->pos0[0];
    fresh = fresh && p->pos0[r] == 0;
    ctx += p->pos0[r] + p->lens[r];
  }
  CG_TRY(grow(c, ST_BF16, ctx * kvw, &X.kv, &X.kv_n));
  char* kv = (char*)X.kv->data();
  if (fresh) a.c_out = X.cpk->data();
  CG_TRY(k_launch_latent_prep(c, a));
  if (fresh) {
    CG_TRY(lin(D, X.cpk->data(), L.Lw, rd.M, L.w_kv, 0, kvw, kv, kvw, 1));
  } else {
    int64_t at = 0;
    for (int r = 0; r < R; ++r) {
      const int64_t n = p->pos0[r] + p->lens[r];
      CG_TRY(lin(D, (const char*)a.cache + (size_t)p->slots[r] * a.Tmax * L.Lw * es, L.Lw, n, L.w_kv, 0, kvw, kv + (size_t)at * kvw * es, kvw,
                 1));
      at += n;
    }
  }
  int64_t tok = 0, at = 0;
  for (int r = 0; r < (equal ? 1 : R); ++r) {
    AttnArgs t;
    t.q = (const __nv_bfloat16*)a.q_out + tok * a.H * Dp;
    t.k_cache = (const __nv_bfloat16*)kv + at * kvw;
    t.v_cache = t.k_cache + a.H * Dp;
    t.out = (__nv_bfloat16*)a.att + tok * L.Ko;
    t.B = equal ? R : 1; t.S = p->lens[r]; t.pos0 = p->pos0[r]; t.Tmax = t.pos0 + t.S;
    t.pos_dev = nullptr;
    t.nh = t.nkv = a.H; t.d = (int)Dp;
    t.window = 0; t.softcap = 0.f; t.scratch = nullptr;
    t.kv_ld = kvw; t.scale = a.scale;
    CG_TRY(k_launch_attn_prefill(c, t));
    tok += t.S;
    at += t.Tmax;
  }
  return CG_OK;
}

void recurrent_base(cg_decoder* D, const MixedLayer& L, MixedRun& run, const RowsDev& rd, RecurBase* a) {
  MixedModel& X = *D->mixed;
  a->delta = L.delta() ? 1 : 0;
  if (L.key_decay()) {
    a->key_decay = 1; a->zs = L.zs;
    a->coef = (const float*)L.coef->data(); a->z_bias = (const float*)L.dt_bias->data();
    a->z_sign = a->delta ? 1.f : -1.f;
    a->linear = a->delta ? 0 : 1;
    if (!a->delta) a->q_scale = (float)(1.0 / std::sqrt((double)L.dk));
  }
  a->H = L.H; a->KH = L.KH; a->dk = L.dk; a->dv = L.dv; a->dvs = L.dvs; a->C = L.C; a->taps = L.k.conv;
  a->q_off = L.q_off; a->k_off = L.k_off; a->v_off = L.v_off; a->qs = L.qs; a->vs = L.vs;
  a->conv_w = L.conv_w ? (const float*)L.conv_w->data() : nullptr;
  a->conv_b = L.conv_b ? (const float*)L.conv_b->data() : nullptr;
  a->tail = run.tail ? (float*)run.tail->data() : nullptr;
  a->a_log = L.a_log ? (const float*)L.a_log->data() : nullptr;
  a->dt_bias = L.dt_bias ? (const float*)L.dt_bias->data() : nullptr;
  a->log_decay = L.log_decay ? (const float*)L.log_decay->data() : nullptr;
  a->dskip = L.dskip ? (const float*)L.dskip->data() : nullptr;
  a->S = (float*)run.state->data();
  a->gl = (float*)(a->key_decay ? X.z : X.gl)->data(); a->co = (float*)X.co->data();
  a->o = (float*)X.ro->data();
  a->rows = rd;
}

// Prompts in a bf16 context run in chunks on the tensor cores, from bf16 projections that the mixer makes itself
bool in_chunks(const MixedLayer& L, const Portion* p) { return L.chunked && p && p->max_len >= 8; }

int lru_layer(cg_decoder* D, const MixedLayer& L, MixedRun& run, const RowsDev& rd, const Portion* p, const Chunks* ch, Rows in, Rows out) {
  MixedModel& X = *D->mixed;
  LruArgs a{};
  const bool bf = in_chunks(L, p);
  if (bf) {
    in.p = X.proj->data();
    in.ld = L.Np;
    CG_TRY(lin(D, X.xn->data(), X.Wp, rd.M, L.w_in, L.in_row, L.Np, in.p, in.ld, 1));
  }
  a.in_bf16 = bf ? 1 : 0;
  a.y = in.p; a.x = (const char*)in.p + (size_t)L.x_off * (bf ? 2 : 4); a.ldx = in.ld;
  a.yb = (const float*)L.yb->data(); a.xb = (const float*)L.xb->data();
  a.W = L.C; a.blocks = L.H; a.taps = L.k.conv;
  a.conv_w = (const float*)L.conv_w->data(); a.conv_b = (const float*)L.conv_b->data();
  a.ra = L.ra->data(); a.ri = L.ri->data();
  a.ra_b = (const float*)L.ra_b->data(); a.ri_b = (const float*)L.ri_b->data();
  a.f = (const float*)L.coef->data();
  a.S = (float*)run.state->data(); a.tail = (float*)run.tail->data();
  a.u = X.u->data(); a.a = (float*)X.lru_a->data(); a.b = (float*)X.lru_b->data();
  a.out = out.p; a.ld_out = out.ld; a.out_bf16 = X.f32 ? 0 : 1;
  a.rows = rd;
  if (ch) { a.chunk_tok = ch->tok; a.chunk_len = ch->len; a.n_chunks = ch->n; }
  return !p || p->max_len == 1 ? k_launch_lru_decode(D->c, a) : k_launch_lru_prompt(D->c, a);
}

// One token per row: one kernel.  Chunks take bf16 projections made here (the decays' and step sizes'
// projections stay f32; lightning's queries, keys and values pass silu in the GEMM).  Otherwise token by token.
int recurrent_layer(cg_decoder* D, const MixedLayer& L, MixedRun& run, const RowsDev& rd, const Portion* p, const Chunks* ch, Rows in,
                    Rows out) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int64_t M = rd.M, K = X.Wp;
  const bool lightning = L.k.mixer == CG_MIX_LIGHTNING, delta = L.delta(), gla = L.k.mixer == CG_MIX_GLA;
  GatedNorm n;
  n.H = L.H; n.dv = L.dv; n.dvs = L.dvs;
  n.groups = delta || gla ? L.H : lightning ? 1 : L.k.norm_groups;
  n.shared_gain = delta || gla; n.gate_first = !delta && !gla && !lightning; n.sigmoid = lightning || L.k.mixer == CG_MIX_CHANNEL_DELTA;
  n.o = (const float*)X.ro->data();
  n.norm = (const float*)L.norm->data(); n.eps = D->cfg.rms_eps;
  n.att = out.p; n.ld_att = out.ld; n.att_bf16 = X.f32 ? 0 : 1;
  n.M = M;
  if (in_chunks(L, p)) {
    ChunkArgs a;
    recurrent_base(D, L, run, rd, &a);
    a.chunk_tok = ch->tok; a.chunk_len = ch->len; a.row_chunk = ch->row_chunk; a.n_chunks = ch->n;
    a.DKp = (int)up16(L.dk); a.dvp = L.dvs;
    a.q = (__nv_bfloat16*)X.qkv->data();
    a.T = nullptr;
    if (L.key_decay()) {
      CG_TRY(grow(c, ST_BF16, (int64_t)ch->n * L.H * channel_scratch(L.dk, a.delta), &X.tinv, &X.tinv_n));
      CG_TRY(grow(c, ST_F32, (int64_t)ch->n * L.H * (L.dk <= 64 ? 64 : 128), &X.decayed, &X.decayed_n));
      a.T = (__nv_bfloat16*)X.tinv->data();
      a.decayed = (float*)X.decayed->data();
    }
    if (gla) {
      // queries, keys, values, gate and the first factor of the decays are one GEMM
      __nv_bfloat16* pb = (__nv_bfloat16*)X.proj->data();
      CG_TRY(lin(D, X.xn->data(), K, M, L.w_in, L.in_row, L.Np, pb, L.Np, 1));
      CG_TRY(lin(D, pb + L.a1_off, L.Np, M, L.w_a2, 0, L.H * L.zs, X.z->data(), (int64_t)L.H * L.zs));
      a.q = pb + L.q_off; a.k = pb + L.k_off; a.v = pb + L.v_off;
      a.ldq = a.ldv = L.Np;
      a.proj = nullptr; a.ldp = 0; a.small = nullptr; a.ld_small = 0; a.rq = a.rk = nullptr;
      CG_TRY(k_launch_chunk_recurrence(c, a));
      n.gate = pb + L.gate_off; n.ldg = L.Np; n.gate_bf16 = 1;
      return k_launch_gated_norm(c, n);
    }
    if (lightning) {
      const int64_t ng = L.Np - L.C;
      __nv_bfloat16* gate = (__nv_bfloat16*)X.proj->data();
      CG_TRY(lin(D, X.xn->data(), K, M, L.w_in, L.in_row, L.C, a.q, L.C, 5));
      CG_TRY(lin(D, X.xn->data(), K, M, L.w_in, L.in_row + L.C, ng, gate, ng, 1));
      a.k = a.q + L.k_off; a.v = a.q + L.v_off;
      a.ldq = a.ldv = L.C;
      a.proj = nullptr; a.ldp = 0; a.small = nullptr; a.ld_small = 0; a.rq = a.rk = nullptr;
      CG_TRY(k_launch_chunk_recurrence(c, a));
      n.gate = gate; n.ldg = ng; n.gate_bf16 = 1;
      return k_launch_gated_norm(c, n);
    }
    __nv_bfloat16* pb = (__nv_bfloat16*)X.proj->data();
    float* small = (float*)(pb + M * L.small_off);  // both fit where the f32 projection would
    const int64_t ns = L.Np - L.small_off;
    CG_TRY(lin(D, X.xn->data(), K, M, L.w_in, L.in_row, L.small_off, pb, L.small_off, 1));
    CG_TRY(lin(D, X.xn->data(), K, M, L.w_in, L.in_row + L.small_off, ns, small, ns));
    a.proj = pb; a.ldp = L.small_off;
    a.small = small; a.ld_small = ns;
    a.k = a.q + M * L.KH * a.DKp;
    a.v = a.k + M * L.KH * a.DKp;
    a.ldq = (int64_t)L.KH * a.DKp; a.ldv = (int64_t)L.H * a.dvp;
    a.rq = (float*)X.rn->data();
    a.rk = a.rq + M * L.KH;
    if (L.key_decay()) {
      CG_TRY(lin(D, pb + L.a1_off, L.small_off, M, L.w_a2, 0, L.H * L.zs, X.z->data(), (int64_t)L.H * L.zs));
      CG_TRY(lin(D, pb + L.g1_off, L.small_off, M, L.w_g2, 0, L.H * L.dv, X.low_gate->data(), (int64_t)L.H * L.dv, 1));
    } else if (a.delta) {
      CG_TRY(grow(c, ST_BF16, (int64_t)ch->n * L.H * 2 * RECUR_CHUNK * RECUR_CHUNK, &X.tinv, &X.tinv_n));
      a.T = (__nv_bfloat16*)X.tinv->data();
    }
    CG_TRY(k_launch_chunk_recurrence(c, a));
    n.gate = pb + L.gate_off; n.ldg = L.small_off; n.gate_bf16 = 1;
    if (L.key_decay()) { n.gate = X.low_gate->data(); n.ldg = (int64_t)L.H * L.dv; }
    return k_launch_gated_norm(c, n);
  }
  RecurArgs a;
  recurrent_base(D, L, run, rd, &a);
  a.proj = (const float*)in.p; a.ldp = in.ld;
  a.gate_off = L.gate_off; a.small_off = L.small_off;
  a.cv = (float*)X.cv->data(); a.ldc = up8(L.C);
  n.gate = a.proj + L.gate_off; n.ldg = in.ld; n.gate_bf16 = 0;
  if (L.key_decay()) {
    a.a1_off = L.a1_off; a.g1_off = L.g1_off; a.a_rank = L.a_rank; a.g_rank = L.g_rank;
    a.w_bf16 = X.f32 ? 0 : 1;
    a.w_a2 = L.w_a2->data();
    a.w_g2 = L.w_g2 ? L.w_g2->data() : nullptr;
  }
  if ((!p || p->max_len == 1) && recur_decode_supported(L.dk, L.dv)) return k_launch_recur_decode(c, a, n);
  if (L.key_decay()) {
    LowRank r{};
    r.ldx = a.ldp; r.w_bf16 = a.w_bf16;
    r.x = a.proj + a.a1_off; r.w = a.w_a2; r.N = L.H * L.zs; r.R = a.a_rank;
    r.coef = a.coef; r.bias = a.z_bias; r.zs = L.zs; r.sign = a.z_sign;
    r.out = a.gl;
    CG_TRY(k_launch_low_rank(c, r, M));
    if (a.w_g2) {
      r.x = a.proj + a.g1_off; r.w = a.w_g2; r.N = L.H * L.dv; r.R = a.g_rank;
      r.coef = r.bias = nullptr;
      r.out = (float*)X.low_gate->data();
      CG_TRY(k_launch_low_rank(c, r, M));
      n.gate = r.out; n.ldg = r.N;
    }
  }
  CG_TRY(k_launch_recur_steps(c, a));
  return k_launch_gated_norm(c, n);
}

// y = the layer's mixer, or the sum of its two, of the rows xn.  The f32 projections of both are one GEMM
// unless one of them makes its own.
int mixer(cg_decoder* D, const MixedLayer& L, MixedRun& run, const RowsDev& rd, const Portion* p, const Chunks* ch) {
  MixedModel& X = *D->mixed;
  const int64_t M = rd.M, Ko = L.out_width();
  if (L.k.mixer == CG_MIX_LATENT) {
    CG_TRY(latent_layer(D, L, run, rd, p));
  } else {
    const size_t es = storage_bytes(X.act_storage());
    const bool joint = L.beside && !in_chunks(L, p) && !in_chunks(*L.beside, p);
    for (int side = 0; side < (L.beside ? 2 : 1); ++side) {
      const MixedLayer& m = side ? *L.beside : L;
      MixedRun& r = side ? *run.beside : run;
      Rows in, out;
      out.p = (char*)X.att->data() + (size_t)m.out_col * es; out.ld = Ko;
      if (joint) {
        in.ld = L.in_width();
        in.p = (float*)X.proj->data() + m.in_row;
        if (!side) CG_TRY(lin(D, X.xn->data(), X.Wp, M, L.w_in, 0, in.ld, X.proj->data(), in.ld));
      } else if (!in_chunks(m, p)) {
        in.ld = m.Np;
        in.p = X.proj->data();
        CG_TRY(lin(D, X.xn->data(), X.Wp, M, L.w_in, m.in_row, m.Np, in.p, m.Np));
      }
      if (m.k.mixer == CG_MIX_ATTENTION) CG_TRY(attention_layer(D, m, r, rd, p, in, out));
      else if (m.lru()) CG_TRY(lru_layer(D, m, r, rd, p, ch, in, out));
      else CG_TRY(recurrent_layer(D, m, r, rd, p, ch, in, out));
    }
  }
  if (L.k.out_norm) {
    // a result each, behind one another in y2
    for (int side = 0; side < 2; ++side) {
      const MixedLayer& m = side ? *L.beside : L;
      const char* at = (const char*)X.att->data() + (size_t)m.out_col * storage_bytes(X.act_storage());
      CG_TRY(lin(D, at, Ko, M, m.w_o, 0, X.Wp, (float*)X.y2->data() + side * M * X.Wp, X.Wp));
    }
    return CG_OK;
  }
  if (L.ff_col >= 0) CG_TRY(gelu_units(D, L, M, Rows{(char*)X.att->data() + (size_t)L.ff_col * storage_bytes(X.act_storage()), Ko}));
  return lin(D, X.att->data(), Ko, M, L.w_o, 0, X.Wp, X.y->data(), X.Wp);
}

// room for the residual streams of all layer runs of M tokens
int keep_room(cg_decoder* D, int64_t M) {
  MixedModel& X = *D->mixed;
  drop(X.kept);
  int64_t d3[3] = {(int64_t)X.runs.size(), M, D->H};
  return new_tensor(D->c, CG_F32, ST_F32, d3, 3, &X.kept);
}

// The walk of designs without post-norms: sublayer by sublayer, each update preparing the next one's
// normed input in xn.
int walk_streams(cg_decoder* D, const RowsDev& rd, const uint32_t* tokens, const Portion* p, const Chunks* ch) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int64_t M = rd.M, Wp = X.Wp;
  const int bf = X.f32 ? 0 : 1;
  const size_t nruns = X.runs.size();
  StreamUpdate base;
  base.ns = X.streams;
  base.x = (float*)X.x->data(); base.ldx = Wp; base.eps = D->cfg.rms_eps; base.W = (int)D->H;
  // what the update leaves for sublayer q of run i
  auto hand_on = [&](StreamUpdate& u, size_t i, int q) {
    if (i >= nruns) return;
    const MixedLayer& L = X.layers[X.runs[i].layer];
    u.in_w = (const float*)L.hc_in[q]->data();
    u.g = (const float*)(q ? L.n2 : L.n1)->data();
    u.out = X.xn->data(); u.ldo = Wp;
  };
  auto update = [&](const MixedLayer& L, int q) {
    StreamUpdate u = base;
    u.mix = (const float*)L.hc_mix[q]->data(); u.out_w = (const float*)L.hc_out[q]->data();
    if (q && L.k.experts) {
      u.y = (const float*)X.m_y->data(); u.ldy = Wp;
      u.pos = (const int32_t*)X.m_pos->data(); u.wts = (const float*)X.m_wts->data(); u.top = L.k.top_k;
    } else {
      u.y = (const float*)X.y->data(); u.ldy = Wp;
    }
    return u;
  };
  {
    StreamUpdate u = base;
    u.tokens = tokens; u.table = D->embed->data(); u.table_bf16 = D->embed->storage == ST_BF16; u.vocab = D->cfg.vocab;
    u.scale = X.embed_scale;
    hand_on(u, 0, 0);
    CG_TRY(k_launch_stream_update(c, u, M, bf));
  }
  for (size_t i = 0; i < nruns; ++i) {
    MixedRun& run = X.runs[i];
    const MixedLayer& L = X.layers[run.layer];
    CG_TRY(mixer(D, L, run, rd, p, ch));
    StreamUpdate u = update(L, 0);
    if (L.k.ffn) {
      hand_on(u, i, 1);
      CG_TRY(k_launch_stream_update(c, u, M, bf));
      if (L.k.experts) CG_TRY(experts_ff(D, L, M));
      else CG_TRY(dense_ff(D, L, M));
      u = update(L, 1);
    }
    hand_on(u, i + 1, 0);
    if (X.keep && p) {
      if (i == 0) CG_TRY(keep_room(D, M));
      u.sum = (float*)X.kept->data() + (int64_t)i * M * D->H; u.ld_sum = D->H;
    }
    CG_TRY(k_launch_stream_update(c, u, M, bf));
  }
  return CG_OK;
}

// The walk of designs whose sublayers run side by side on one norm.  Per layer: its branches are added, then
// the input for the token itself, and one pass keeps the result, averages over all results so far and
// prepares the next layer's normed input.
int walk_parallel(cg_decoder* D, const RowsDev& rd, const uint32_t* tokens, const Portion* p, const Chunks* ch) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int64_t M = rd.M, Wp = X.Wp;
  const int bf = X.f32 ? 0 : 1;
  auto data = [](const cg_tensor* t) { return t ? (const float*)t->data() : nullptr; };
  DepthUpdate base;
  base.x = (float*)X.x->data(); base.ldx = Wp; base.eps = D->cfg.rms_eps; base.W = (int)D->H;
  if (X.depth) { base.depth = (float*)X.depth->data(); base.depth_stride = M * Wp; }
  auto hand_on = [&](DepthUpdate& u, size_t i) {
    if (i >= X.runs.size()) return;
    u.g = data(X.layers[X.runs[i].layer].n1);
    u.out = X.xn->data(); u.ldo = Wp;
  };
  {
    DepthUpdate u = base;
    u.tokens = tokens; u.table = D->embed->data(); u.table_bf16 = D->embed->storage == ST_BF16; u.vocab = D->cfg.vocab;
    u.scale = X.embed_scale;
    hand_on(u, 0);
    CG_TRY(k_launch_depth_update(c, u, M, bf));
  }
  for (size_t i = 0; i < X.runs.size(); ++i) {
    MixedRun& run = X.runs[i];
    const MixedLayer& L = X.layers[run.layer];
    BranchSum s;
    s.x = (float*)X.x->data(); s.ldx = Wp; s.eps = D->cfg.rms_eps; s.W = (int)D->H;
    s.ldy = Wp;
    CG_TRY(mixer(D, L, run, rd, p, ch));
    if (L.k.out_norm) {
      s.normed[0] = (const float*)X.y2->data(); s.normed[1] = s.normed[0] + M * Wp;
      s.gain[0] = data(L.out_gain); s.gain[1] = data(L.beside->out_gain);
    } else {
      s.y = (const float*)X.y->data();
    }
    if (L.k.experts) {
      CG_TRY(experts_ff(D, L, M));
      s.ye = (const float*)X.m_y->data(); s.pos = (const int32_t*)X.m_pos->data(); s.wts = (const float*)X.m_wts->data(); s.top = L.k.top_k;
    } else if (L.k.ffn) {
      if (L.ff_col < 0) {
        CG_TRY(dense_ff(D, L, M));
        s.y = (const float*)X.y->data();
      }
      s.y_bias = data(L.down_bias);
    }
    if (X.side_p) { s.copy = X.xn->data(); s.ld_copy = Wp; }
    CG_TRY(k_launch_branch_sum(c, s, M, bf));
    DepthUpdate u = base;
    if (X.side_p) {
      CG_TRY(lin(D, X.xn->data(), Wp, M, L.side_gate, 0, X.side_p, X.side_z->data(), X.side_p));
      TokenGate g{};
      g.tokens = tokens; g.vocab = D->cfg.vocab;
      g.table = X.side_embed->data(); g.ld_table = (int64_t)D->cfg.token_side * X.layers.size(); g.off = (int64_t)i * D->cfg.token_side;
      g.z = (const float*)X.side_z->data(); g.ldz = X.side_p; g.n = D->cfg.token_side;
      g.out = X.side_h->data(); g.ldo = X.side_p;
      CG_TRY(k_launch_token_gate(c, g, M, bf));
      CG_TRY(lin(D, X.side_h->data(), X.side_p, M, L.side_proj, 0, Wp, X.y->data(), Wp));
      u.y = (const float*)X.y->data(); u.ldy = Wp; u.y_gain = data(L.side_norm);
    }
    u.average = data(L.average); u.n = (int)i + 1;
    hand_on(u, i + 1);
    if (X.keep && p) {
      if (i == 0) CG_TRY(keep_room(D, M));
      u.kept = (float*)X.kept->data() + (int64_t)i * M * D->H; u.ld_kept = D->H;
    }
    CG_TRY(k_launch_depth_update(c, u, M, bf));
  }
  return CG_OK;
}

// out[dst[i]] = the final norm of packed token pick[i]'s residual stream
int final_rows(cg_decoder* D, const int32_t* pick, const int32_t* dst, int64_t n, void* out) {
  MixedModel& X = *D->mixed;
  auto fill = [&](auto& u) {
    u.x = (float*)X.x->data(); u.ldx = X.Wp; u.eps = D->cfg.rms_eps; u.W = (int)D->H;
    u.pick = pick; u.dst = dst;
    u.out = out; u.ldo = X.Wp;
  };
  if (X.sandwich) {
    RowUpdate u;
    fill(u);
    u.g2 = (const float*)D->ln_f->data();
    u.b2 = X.ln_f_bias ? (const float*)X.ln_f_bias->data() : nullptr;
    u.centred = D->cfg.layer_norm;
    return k_launch_row_update(D->c, u, n, X.f32 ? 0 : 1);
  }
  StreamUpdate u;
  fill(u);
  u.ns = X.streams;
  u.g = (const float*)D->ln_f->data();
  return k_launch_stream_update(D->c, u, n, X.f32 ? 0 : 1);
}

// Embedding and all layer runs of one batch; x holds the residual stream afterwards.  p is null in
// decode steps (one token per row).
int walk(cg_decoder* D, const RowsDev& rd, const uint32_t* tokens, const Portion* p, const Chunks* ch) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  if (X.parallel) return walk_parallel(D, rd, tokens, p, ch);
  if (!X.sandwich) return walk_streams(D, rd, tokens, p, ch);
  const int64_t M = rd.M, W = D->H, Wp = X.Wp;
  const int bf = X.f32 ? 0 : 1;
  char* cat_lo = X.loop ? (char*)X.xcat->data() : nullptr;
  char* cat_hi = X.loop ? cat_lo + (size_t)Wp * storage_bytes(X.act_storage()) : nullptr;
  const size_t nruns = X.runs.size();
  auto data = [](const cg_tensor* t) { return t ? (const float*)t->data() : nullptr; };
  // the next sublayer's input rows: the stream, normed if the design has norms there
  auto input_rows = [&](RowUpdate& u, const cg_tensor* g, const cg_tensor* b) {
    u.out = X.xn->data(); u.ldo = Wp; u.g2 = data(g); u.b2 = data(b);
  };
  // what the row update leaves for run i: its input, or the first half of a pass's input rows
  auto hand_on = [&](RowUpdate& u, size_t i) {
    if (i >= nruns) return;
    const MixedLayer& L = X.layers[X.runs[i].layer];
    if (X.runs[i].starts_pass) { u.out = cat_lo; u.ldo = 2 * Wp; u.g2 = nullptr; }
    else input_rows(u, L.n1, L.n1_bias);
  };
  RowUpdate base;
  base.centred = D->cfg.layer_norm;
  base.x = (float*)X.x->data(); base.ldx = Wp; base.eps = D->cfg.rms_eps; base.W = (int)W;
  {
    RowUpdate u = base;
    u.tokens = tokens; u.table = D->embed->data(); u.table_bf16 = D->embed->storage == ST_BF16; u.vocab = D->cfg.vocab;
    u.scale = X.embed_scale;
    u.g1 = X.embed_norm ? (const float*)X.embed_norm->data() : nullptr;
    u.x0 = cat_hi; u.ld0 = 2 * Wp;
    hand_on(u, 0);
    CG_TRY(k_launch_row_update(c, u, M, bf));
  }
  for (size_t i = 0; i < nruns; ++i) {
    MixedRun& run = X.runs[i];
    const MixedLayer& L = X.layers[run.layer];
    if (run.starts_pass) {
      CG_TRY(lin(D, cat_lo, 2 * Wp, M, X.w_loop, 0, Wp, X.y->data(), Wp));
      RowUpdate u = base;
      u.y = (const float*)X.y->data(); u.ldy = Wp;
      input_rows(u, L.n1, L.n1_bias);
      CG_TRY(k_launch_row_update(c, u, M, bf));
    }
    CG_TRY(mixer(D, L, run, rd, p, ch));
    RowUpdate u = base;
    u.y = (const float*)X.y->data(); u.ldy = Wp; u.add = 1;
    u.g1 = data(L.n1b); u.b1 = data(L.n1b_bias);
    if (L.k.ffn) {
      input_rows(u, L.n2, L.n2_bias);
      CG_TRY(k_launch_row_update(c, u, M, bf));
      if (L.k.experts) {
        CG_TRY(experts_ff(D, L, M));
        u.ye = (const float*)X.m_y->data(); u.ldye = Wp;
        u.pos = (const int32_t*)X.m_pos->data(); u.top = L.k.top_k;
        u.wts = L.k.weigh_input ? nullptr : (const float*)X.m_wts->data();
      }
      if (L.Fd) CG_TRY(dense_ff(D, L, M));
      else u.y = nullptr;
      u.g1 = data(L.n2b); u.b1 = data(L.n2b_bias);
      u.out = nullptr; u.g2 = u.b2 = nullptr;
    }
    hand_on(u, i + 1);
    CG_TRY(k_launch_row_update(c, u, M, bf));
    if (X.keep && p) {
      if (i == 0) CG_TRY(keep_room(D, M));
      CG_CUDA(c, cudaMemcpy2DAsync((float*)X.kept->data() + (int64_t)i * M * W, (size_t)W * 4, X.x->data(), (size_t)Wp * 4, (size_t)W * 4,
                                   (size_t)M, cudaMemcpyDeviceToDevice, c->core->stream));
    }
  }
  return CG_OK;
}

int bad_size(cg_decoder* D, int li, const char* what) {
  return fail(D->c, CG_ERR_INVALID, "decoder: layer " + std::to_string(li) + ": " + what);
}

}  // namespace

int mixed_create(cg_decoder* D, const cg_layer_config* layers, int n_layers, const cg_loop_config* loop) {
  auto* X = new MixedModel();
  D->mixed = X;
  X->f32 = D->c->precision == CG_PREC_F32;
  X->Wp = up8(D->H);
  X->sandwich = D->cfg.post_norms != 0;
  X->parallel = D->cfg.parallel_sublayers != 0;
  X->streams = std::max(D->cfg.streams, 1);
  if (D->cfg.embed_scale != 0.f) X->embed_scale = D->cfg.embed_scale;
  if (D->cfg.streams < 0 || D->cfg.streams > MAX_STREAMS) return fail(D->c, CG_ERR_UNSUPPORTED, "decoder: at most 16 streams");
  if (X->sandwich && (D->cfg.streams || D->cfg.norm_plus_one))
    return fail(D->c, CG_ERR_UNSUPPORTED, "decoder: post-norms go with one stream and plain gains");
  if (!X->sandwich && (D->cfg.embed_norm || D->cfg.loop_input || D->cfg.layer_norm || (D->cfg.residual_mult != 0.f && D->cfg.residual_mult != 1.f) ||
                       (D->cfg.logit_scale != 0.f && D->cfg.logit_scale != 1.f)))
    return fail(D->c, CG_ERR_UNSUPPORTED, "decoder: a normed embedding, looped inputs, layer norms, residual and logit factors go with post-norms");
  if (X->parallel && (X->sandwich || D->cfg.streams || D->cfg.norm_plus_one || loop))
    return fail(D->c, CG_ERR_UNSUPPORTED, "decoder: sublayers side by side go with one stream, plain gains and no loop");
  if (!X->parallel && (D->cfg.depth_average || D->cfg.token_side))
    return fail(D->c, CG_ERR_UNSUPPORTED, "decoder: averages over depth and token inputs go with sublayers side by side");
  if (D->cfg.token_side < 0) return fail(D->c, CG_ERR_INVALID, "decoder: token input size");
  X->side_p = up8(D->cfg.token_side);
  X->layers.resize(n_layers);
  auto take_mixer = [&](int i, MixedLayer& L, bool two) -> int {
    const cg_layer_config& k = L.k;
    if (k.heads < 1 || k.vdim < 1) return bad_size(D, i, "sizes must be positive");
    X->recurrent = X->recurrent || L.recurrent();
    if (k.mixer == CG_MIX_ATTENTION) {
      if (k.dim < 1 || k.kv_heads < 1 || k.heads % k.kv_heads || k.window < 0 || k.keep_first < 0 || k.rot_dim < 0 || k.rot_dim % 2 ||
          k.rot_dim > k.dim || (k.rot_dim && !(k.rot_base > 0)) || !(k.scale > 0) || k.qk_norm < 0 || k.qk_norm > 2 ||
          (k.qk_norm == 1 && k.rot_half && k.rot_dim) || k.gate < 0 || k.gate > 2 || k.q_temp_every < 0)
        return bad_size(D, i, "attention sizes");
      if (!k.window) L.k.keep_first = 0;
    } else if (k.mixer == CG_MIX_LATENT) {
      if (k.dim < 1 || k.rot_dim < 0 || k.rot_dim % 2 || k.kv_rank < 1 || (k.rot_dim && !(k.rot_base > 0)) || two)
        return bad_size(D, i, "latent attention sizes");
    } else if (k.mixer == CG_MIX_DELTA || k.mixer == CG_MIX_CHANNEL_DELTA) {
      if (k.dim < 1 || k.kv_heads < 1 || k.heads % k.kv_heads || k.conv < 1) return bad_size(D, i, "delta rule sizes");
    } else if (k.mixer == CG_MIX_SSD) {
      if (k.state < 1 || k.groups < 1 || k.heads % k.groups || k.norm_groups < 1 || (k.heads * k.vdim) % k.norm_groups || k.conv < 1)
        return bad_size(D, i, "state space sizes");
    } else if (k.mixer == CG_MIX_LIGHTNING) {
      if (k.dim < 1 || !k.decay) return bad_size(D, i, "lightning attention sizes");
      L.k.conv = 0;
      L.decay.assign(k.decay, k.decay + k.heads);
      for (double x : L.decay)
        if (!(x >= 0. && x <= 1.)) return bad_size(D, i, "decays must be in [0, 1]");
    } else if (k.mixer == CG_MIX_GLA) {
      if (k.dim < 1 || !(k.tau > 0)) return bad_size(D, i, "gated linear attention sizes");
      L.k.conv = 0;
    } else if (k.mixer == CG_MIX_LRU) {
      if (k.conv < 1) return bad_size(D, i, "recurrent block sizes");
      L.chunked = !X->f32;
    } else return bad_size(D, i, "unknown mixer");
    L.k.decay = nullptr;
    L.k.beside = nullptr;
    return CG_OK;
  };
  for (int i = 0; i < n_layers; ++i) {
    const cg_layer_config& k = layers[i];
    X->layers[i].k = k;
    if (k.weights_of < 0 || k.weights_of > n_layers || k.weights_of == i + 1 || (k.weights_of && layers[k.weights_of - 1].weights_of))
      return bad_size(D, i, "weights of no layer");
    if (k.ffn < 0 || k.shared_ffn < 0) return bad_size(D, i, "sizes must be positive");
    if (k.shared_ffn && (!k.experts || !X->sandwich)) return bad_size(D, i, "a shared expert goes with experts and post-norms");
    if (X->parallel && k.weights_of) return bad_size(D, i, "weights of another layer go with sublayers one after the other");
    if (k.out_norm && (!X->parallel || !k.beside)) return bad_size(D, i, "norms of two mixers' results go with sublayers side by side");
    if (k.weigh_input && !X->sandwich) return bad_size(D, i, "weighted inputs of experts go with post-norms");
    if (k.ffn && k.experts) {
      if (k.experts < 0 || k.experts > 1024 || k.top_k < 1 || k.top_k > 32 || k.top_k > k.experts)
        return bad_size(D, i, "1 to 1024 experts, at most 32 per token");
      if (k.act < CG_ACT_SILU || k.act > CG_ACT_RELU2 || (k.act == CG_ACT_BOUNDED && !(k.act_limit > 0)))
        return bad_size(D, i, "activation of the experts");
    } else if (k.ffn && k.act != CG_ACT_SILU && k.act != CG_ACT_GELU && k.act != CG_ACT_RELU2 && !(k.act == CG_ACT_GELU1 && X->parallel)) {
      return bad_size(D, i, "activation of the feed-forward");
    }
    if (!k.ffn) X->layers[i].k.experts = X->layers[i].k.shared_ffn = 0;
    if (k.beside) {
      X->layers[i].beside = std::make_unique<MixedLayer>();
      X->layers[i].beside->k = *k.beside;
      CG_TRY(take_mixer(i, *X->layers[i].beside, true));
    }
    CG_TRY(take_mixer(i, X->layers[i], k.beside != nullptr));
  }
  const bool looped = loop && loop->times > 0 && loop->stop > loop->start;
  if (looped && (loop->start < 0 || loop->stop > n_layers)) return fail(D->c, CG_ERR_INVALID, "decoder: loop out of range");
  X->loop = looped && D->cfg.loop_input;
  auto add = [&](int i, bool starts) {
    MixedRun r;
    r.layer = layers[i].weights_of ? layers[i].weights_of - 1 : i;
    r.starts_pass = starts;
    if (X->layers[r.layer].beside) r.beside = std::make_unique<MixedRun>();
    X->runs.push_back(std::move(r));
  };
  const int a = looped ? loop->start : n_layers, b = looped ? loop->stop : n_layers;
  for (int i = 0; i < a; ++i) add(i, false);
  for (int t = 0; looped && t < loop->times; ++t)
    for (int i = a; i < b; ++i) add(i, X->loop && i == a);
  for (int i = b; i < n_layers; ++i) add(i, false);
  X->open.assign(D->cfg.max_batch, 0);
  X->pos.assign(D->cfg.max_batch, 0);
  return CG_OK;
}

void mixed_destroy(cg_decoder* D) {
  MixedModel* X = D->mixed;
  if (!X) return;
  auto drop_layer = [](MixedLayer& L) {
    for (cg_tensor** t : {&L.n1, &L.n1b, &L.n2, &L.n2b, &L.n1_bias, &L.n1b_bias, &L.n2_bias, &L.n2b_bias, &L.log_decay, &L.w_in, &L.w_o, &L.w_gu, &L.w_down, &L.c_gain, &L.uk, &L.uv, &L.w_kv, &L.cos_t,
                          &L.sin_t, &L.conv_w, &L.conv_b, &L.a_log, &L.dt_bias, &L.dskip, &L.norm, &L.q_gain, &L.k_gain, &L.sink,
                          &L.router, &L.correction, &L.we_gate, &L.we_up, &L.we_down, &L.up_bias, &L.down_bias, &L.out_gain, &L.average,
                          &L.side_gate, &L.side_proj, &L.side_norm, &L.q_temp, &L.bias, &L.coef, &L.w_a2, &L.w_g2, &L.ra, &L.ri, &L.ra_b,
                          &L.ri_b, &L.xb, &L.yb})
      drop(*t);
    for (int q = 0; q < 2; ++q) { drop(L.hc_in[q]); drop(L.hc_out[q]); drop(L.hc_mix[q]); }
  };
  auto drop_run = [](MixedRun& r) { drop(r.cache); drop(r.cache_v); drop(r.state); drop(r.tail); };
  for (MixedLayer& L : X->layers) {
    if (L.beside) drop_layer(*L.beside);
    drop_layer(L);
  }
  for (MixedRun& r : X->runs) {
    if (r.beside) drop_run(*r.beside);
    drop_run(r);
  }
  for (cg_tensor** t : {&X->embed_norm, &X->ln_f_bias, &X->w_loop, &X->tab_run, &X->tab_dec, &X->x, &X->xn, &X->xcat, &X->y, &X->proj, &X->cv, &X->gl,
                        &X->co, &X->ro, &X->att, &X->hact, &X->gu, &X->q, &X->cpk, &X->tok, &X->xw, &X->kept, &X->qkv, &X->rn,
                        &X->tinv, &X->kv, &X->lat, &X->m_logits, &X->m_ids, &X->m_wts, &X->m_pos, &X->m_tiles, &X->m_xg, &X->m_h,
                        &X->m_y, &X->z, &X->low_gate, &X->u, &X->lru_a, &X->lru_b, &X->y2, &X->depth, &X->side_z, &X->side_h, &X->side_embed, &X->decayed})
    drop(*t);
  delete X;
  D->mixed = nullptr;
}

int mixed_finalize(cg_decoder* D) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int64_t W = D->H;
  const int st = X.act_storage();
  const bool pre = D->cfg.post_norms != 2;
  const float mult = D->cfg.residual_mult != 0.f ? D->cfg.residual_mult : 1.f;
  for (size_t i = 0; i < X.layers.size(); ++i) {
    MixedLayer& L = X.layers[i];
    if (L.k.weights_of) continue;
    const std::string l = "l" + std::to_string(i) + ".";
    auto norms = [&](const std::string& n, cg_tensor** w, cg_tensor** wb, cg_tensor** after, cg_tensor** after_b) -> int {
      if (pre) CG_TRY(norm_pair(D, n, w, wb));
      return X.sandwich ? norm_pair(D, pre ? n + "b" : n, after, after_b, mult) : CG_OK;
    };
    CG_TRY(norms(l + "norm1", &L.n1, &L.n1_bias, &L.n1b, &L.n1b_bias));
    for (int q = 0; q < (L.k.ffn ? 2 : 1) && !X.sandwich && !X.parallel; ++q) {
      const std::string hc = l + (q ? "hc2." : "hc1.");
      CG_TRY(coefficients(D, hc + "in", X.streams, &L.hc_in[q]));
      CG_TRY(coefficients(D, hc + "out", X.streams, &L.hc_out[q]));
      CG_TRY(coefficients(D, hc + "mix", (int64_t)X.streams * X.streams, &L.hc_mix[q]));
    }
    CG_TRY(L.beside ? finalize_beside(D, L, l + "mix.") : finalize_mixer(D, L, l + "mix."));
    if (L.k.ffn) {
      L.Fp = up8(L.k.ffn);
      if (!X.parallel) CG_TRY(norms(l + "norm2", &L.n2, &L.n2_bias, &L.n2b, &L.n2b_bias));
      if (L.k.experts) CG_TRY(finalize_experts(D, L, l + "mlp."));
      const int64_t F = L.k.experts ? L.k.shared_ffn : L.k.ffn;
      if (F) {
        const std::string ff = l + (L.k.experts ? "mlp.shared." : "mlp.");
        const bool gated = L.k.act != CG_ACT_RELU2 && L.k.act != CG_ACT_GELU1;
        L.Fd = up8(F);
        CG_TRY(new2(c, st, (gated ? 2 : 1) * L.Fd, X.Wp, &L.w_gu));
        if (gated) CG_TRY(place_all(D, ff + "gate", F, W, L.w_gu, 0));
        CG_TRY(place_all(D, ff + "up", F, W, L.w_gu, gated ? L.Fd : 0));
        CG_TRY(new2(c, st, X.Wp, L.Fd, &L.w_down));
        CG_TRY(place_all(D, ff + "down", W, F, L.w_down, 0));
        if (L.k.act == CG_ACT_GELU1) {
          CG_TRY(head_gains(D, ff + "up.b", 1, F, L.Fd, &L.up_bias));
          CG_TRY(gains(D, ff + "down.b", W, &L.down_bias));
        }
        if (X.parallel && !L.k.out_norm && L.k.mixer != CG_MIX_LATENT) {
          // the mixer's output and the units side by side: one product adds both sublayers
          const size_t es = storage_bytes(st);
          const int64_t ko = L.out_width();
          Hold both;
          CG_TRY(new2(c, st, X.Wp, ko + L.Fd, &both.t));
          for (int part = 0; part < 2; ++part) {
            const cg_tensor* w = part ? L.w_down : L.w_o;
            const int64_t cols = part ? L.Fd : ko;
            CG_CUDA(c, cudaMemcpy2DAsync((char*)both.t->data() + (size_t)(part ? ko : 0) * es, (size_t)(ko + L.Fd) * es, w->data(), (size_t)cols * es,
                                         (size_t)cols * es, (size_t)X.Wp, cudaMemcpyDeviceToDevice, c->core->stream));
          }
          drop(L.w_o);
          drop(L.w_down);
          L.w_o = both.take();
          L.ff_col = ko;
        }
      }
    }
    if (D->cfg.depth_average) CG_TRY(norm_weight(D, l + "dwa", (int64_t)i + 2, &L.average));
    if (X.side_p) {
      const int64_t n = D->cfg.token_side;
      CG_TRY(new2(c, st, X.side_p, X.Wp, &L.side_gate));
      CG_TRY(place_all(D, l + "side.gate", n, W, L.side_gate, 0));
      CG_TRY(new2(c, st, X.Wp, X.side_p, &L.side_proj));
      CG_TRY(place_all(D, l + "side.proj", W, n, L.side_proj, 0));
      CG_TRY(gains(D, l + "side.norm", W, &L.side_norm));
    }
    // the originals of this layer are no longer needed
    for (auto it = D->params.begin(); it != D->params.end();) {
      if (it->first.compare(0, l.size(), l) == 0) { release(it->second); it = D->params.erase(it); }
      else ++it;
    }
  }
  const int64_t slots = D->cfg.max_batch;
  auto open_run = [&](MixedRun& r, const MixedLayer& L) -> int {
    if (L.k.mixer == CG_MIX_ATTENTION) {
      CG_TRY(new2(c, st, slots * L.k.kv_heads * D->cfg.max_seq, L.Dk, &r.cache));
      CG_TRY(new2(c, st, slots * L.k.kv_heads * D->cfg.max_seq, L.Dv, &r.cache_v));
    } else if (L.k.mixer == CG_MIX_LATENT) {
      CG_TRY(new2(c, st, slots * D->cfg.max_seq, L.Lw, &r.cache));
    } else if (L.lru()) {
      CG_TRY(new2(c, ST_F32, slots, L.C, &r.state));
      CG_TRY(new2(c, ST_F32, slots * L.k.conv, L.C, &r.tail));
    } else {
      CG_TRY(new2(c, ST_F32, slots * L.H * L.dk, L.dvs, &r.state));
      if (L.k.conv) CG_TRY(new2(c, ST_F32, slots * L.k.conv, L.C, &r.tail));
    }
    return CG_OK;
  };
  for (MixedRun& r : X.runs) {
    const MixedLayer& L = X.layers[r.layer];
    CG_TRY(open_run(r, L));
    if (r.beside) CG_TRY(open_run(*r.beside, *L.beside));
  }
  if (X.loop) {
    CG_TRY(new2(c, st, X.Wp, 2 * X.Wp, &X.w_loop));
    CG_TRY(place(D, "loop.in", W, 2 * W, 0, W, 0, W, X.w_loop, 0, 0));
    CG_TRY(place(D, "loop.in", W, 2 * W, 0, W, W, W, X.w_loop, 0, X.Wp));
  }
  if (D->cfg.embed_norm) CG_TRY(norm_weight(D, "embed.norm", W, &X.embed_norm));
  CG_TRY(norm_pair(D, "final.norm", &D->ln_f, &X.ln_f_bias, D->cfg.logit_scale != 0.f ? D->cfg.logit_scale : 1.f));
  CG_TRY(new2(c, st, D->cfg.vocab, W, &D->embed, false));
  CG_TRY(place_all(D, "embed", D->cfg.vocab, W, D->embed, 0));
  if (X.side_p) {
    const int64_t n = (int64_t)D->cfg.token_side * X.layers.size();
    CG_TRY(new2(c, st, D->cfg.vocab, n, &X.side_embed, false));
    CG_TRY(place_all(D, "side.embed", D->cfg.vocab, n, X.side_embed, 0));
  }
  if (D->cfg.tie_embeddings && X.Wp == W) {
    D->head = D->embed;
    D->head->rc++;
  } else {
    CG_TRY(new2(c, st, D->cfg.vocab, X.Wp, &D->head));
    CG_TRY(place_all(D, D->cfg.tie_embeddings ? "embed" : "head", D->cfg.vocab, W, D->head, 0));
  }
  for (auto& kv : D->params) release(kv.second);
  D->params.clear();

  int64_t n = 4;
  CG_TRY(new_tensor(c, CG_U32, ST_U32, &n, 1, &D->state));  // 16 bytes: two int64
  n = slots;
  CG_TRY(new_tensor(c, CG_U32, ST_U32, &n, 1, &D->cur));
  int64_t hd[2] = {slots, D->cfg.max_seq};
  CG_TRY(new_tensor(c, CG_U32, ST_U32, hd, 2, &D->history));
  int64_t ld[3] = {1, slots, D->Vp};
  CG_TRY(new_tensor(c, CG_F32, ST_F32, ld, 3, &D->logits));
  n = 2 * slots;
  CG_TRY(new_tensor(c, CG_U32, ST_U32, &n, 1, &D->best));
  CG_CUDA(c, cudaMemsetAsync(D->best->data(), 0, (size_t)n * 4, c->core->stream));
  n = table_words(slots, slots);
  CG_TRY(new_tensor(c, CG_U32, ST_U32, &n, 1, &X.tab_dec));
  CG_TRY(new2(c, st, slots, X.Wp, &D->xl));
  // split-K partials of problems of at most 64 tokens
  int64_t widest = std::max<int64_t>(X.Wp, D->Vp);
  for (const MixedLayer& L : X.layers)
    widest = std::max({widest, L.in_width(), 2 * L.Fp, 2 * L.Fd, (int64_t)L.k.experts, (int64_t)L.H * L.zs, (int64_t)L.H * L.dv, X.side_p});
  n = X.f32 ? 1 : std::max<int64_t>(8 * 64 * widest, (int64_t)300 * 128 * 256);
  CG_TRY(new_tensor(c, CG_F32, ST_F32, &n, 1, &D->splitk));
  D->splitk_floats = n;
  CG_TRY(ensure_mixed(D, slots));
  CG_TRY(set_state(D, 0, 0));
  D->finalized = true;
  return cg_sync(c);
}

int mixed_reset(cg_decoder* D) {
  MixedModel& X = *D->mixed;
  std::fill(X.open.begin(), X.open.end(), 0);
  std::fill(X.pos.begin(), X.pos.end(), 0);
  X.cur_slots.clear();
  X.tables_current = false;
  D->B = 0;
  return set_state(D, 0, 0);
}

int mixed_run(cg_decoder* D, const std::vector<int>& slots, const std::vector<int>& lens, const uint32_t* tokens, const int32_t* want,
              int n_want, bool greedy, bool new_record, cg_tensor** logits_out) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int R = (int)slots.size();
  if (R < 1 || R > D->cfg.max_batch) return fail(c, CG_ERR_SHAPE, "decoder: rows out of range");
  std::vector<int64_t> first(R + 1, 0);
  std::vector<uint8_t> seen(D->cfg.max_batch, 0);
  int longest = 0;
  for (int r = 0; r < R; ++r) {
    const int s = slots[r];
    if (s < 0 || s >= D->cfg.max_batch || !X.open[s] || seen[s]) return fail(c, CG_ERR_INVALID, "decoder: rows must name open sequences, each once");
    seen[s] = 1;
    if (lens[r] < 1 || X.pos[s] + lens[r] > D->cfg.max_seq) return fail(c, CG_ERR_SHAPE, "decoder: length out of range");
    first[r + 1] = first[r] + lens[r];
    longest = std::max(longest, lens[r]);
  }
  for (int i = 0; i < n_want; ++i)
    if (want[i] < 0 || want[i] >= first[R] || (i && want[i] <= want[i - 1]))
      return fail(c, CG_ERR_INVALID, "decoder: wanted places must be ascending and inside the batch");
  const int64_t generated = greedy && !new_record ? D->generated : 0;
  if (greedy && generated >= D->cfg.max_seq) return fail(c, CG_ERR_SHAPE, "decoder: token history is full");
  X.tables_current = false;
  CG_TRY(set_state(D, 0, greedy ? generated : D->generated));

  const int64_t n_out = n_want + (greedy ? R : 0);
  if (n_out > X.cap_w) {
    CG_TRY(new2(c, X.act_storage(), n_out, X.Wp, &X.xw));
    X.cap_w = n_out;
  }
  // long prompts run in portions, so that the workspace stays bounded
  int64_t Sc = std::max<int64_t>(1, c->opt_prefill_chunk / R);
  if (Sc > 64) Sc = Sc / 64 * 64;
  const bool whole = Sc >= longest;
  for (int64_t p0 = 0; p0 < longest; p0 += Sc) {
    Portion p;
    std::vector<int> row_of;
    std::vector<int64_t> from;
    for (int r = 0; r < R; ++r) {
      const int64_t n = std::min<int64_t>(Sc, lens[r] - p0);
      if (n <= 0) continue;
      p.slots.push_back(slots[r]);
      p.lens.push_back((int)n);
      p.pos0.push_back(X.pos[slots[r]] + p0);
      row_of.push_back(r);
      from.push_back(p.M);
      p.M += n;
      p.max_len = std::max<int>(p.max_len, (int)n);
    }
    CG_TRY(ensure_mixed(D, p.M));
    const uint32_t* toks = tokens;
    if (!whole) {
      for (size_t j = 0; j < row_of.size(); ++j)
        CG_CUDA(c, cudaMemcpyAsync((uint32_t*)X.tok->data() + from[j], tokens + first[row_of[j]] + p0, (size_t)p.lens[j] * 4,
                                   cudaMemcpyDeviceToDevice, c->core->stream));
      toks = (const uint32_t*)X.tok->data();
    }
    // outputs of this portion: (place in the portion, output row)
    std::vector<int32_t> pick, dst;
    int wi = 0;
    for (size_t j = 0; j < row_of.size(); ++j) {
      const int r = row_of[j];
      const int64_t lo = first[r] + p0, hi = lo + p.lens[j];
      while (wi < n_want && want[wi] < lo) ++wi;
      for (; wi < n_want && want[wi] < hi; ++wi) {
        pick.push_back((int32_t)(from[j] + want[wi] - lo));
        dst.push_back(wi);
      }
      if (greedy && p0 + p.lens[j] == lens[r]) {
        pick.push_back((int32_t)(from[j] + p.lens[j] - 1));
        dst.push_back(n_want + r);
      }
    }
    const int64_t tw = table_words((int64_t)row_of.size(), p.M), words = tw + 2 * (int64_t)pick.size();
    if (words > X.tab_run_words) {
      drop(X.tab_run);
      int64_t n = words + words / 4;
      CG_TRY(new_tensor(c, CG_U32, ST_U32, &n, 1, &X.tab_run));
      X.tab_run_words = n;
    }
    RowsDev rd;
    Chunks ch;
    CG_TRY(write_tables(D, p, X.tab_run, &rd, &ch));
    CG_TRY(walk(D, rd, toks, &p, &ch));
    if (!pick.empty()) {
      int32_t* pd = (int32_t*)X.tab_run->data() + tw;
      const size_t np = pick.size();
      CG_CUDA(c, cudaMemcpyAsync(pd, pick.data(), np * 4, cudaMemcpyHostToDevice, c->core->stream));
      CG_CUDA(c, cudaMemcpyAsync(pd + np, dst.data(), np * 4, cudaMemcpyHostToDevice, c->core->stream));
      CG_TRY(final_rows(D, pd, pd + np, (int64_t)np, X.xw->data()));
    }
  }
  for (int r = 0; r < R; ++r) X.pos[slots[r]] += lens[r];
  if (n_want > 0 && logits_out) {
    int64_t d2[2] = {n_want, D->Vp};
    Hold out;
    CG_TRY(new_tensor(c, CG_F32, ST_F32, d2, 2, &out.t));
    CG_TRY(lin(D, X.xw->data(), X.Wp, n_want, D->head, 0, D->Vp, out.t->data(), D->Vp));
    *logits_out = out.take();
  }
  if (greedy) {
    const char* xr = (const char*)X.xw->data() + (size_t)n_want * X.Wp * storage_bytes(X.act_storage());
    float* lg = (float*)D->logits->data();
    CG_TRY(lin(D, xr, X.Wp, R, D->head, 0, D->Vp, lg, D->Vp));
    CG_TRY(k_launch_argmax(c, lg, R, D->Vp, 1, D->cfg.final_softcap, (uint32_t*)D->cur->data(), (uint32_t*)D->history->data(),
                           D->cfg.max_seq, D->count_dev(), D->pos_dev(), 0, (unsigned long long*)D->best->data()));
    CG_TRY(set_state(D, 0, generated + 1));  // (that token is not cached yet)
    X.cur_slots = slots;
    D->B = R;
  }
  return CG_OK;
}

int mixed_prefill(cg_decoder* D, const cg_tensor* tokens, bool fresh) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  if (tokens->tag != CG_U32 || tokens->rank != 2) return fail(c, CG_ERR_SHAPE, "decoder: tokens must be U32 [B, S]");
  const int64_t B = tokens->dims[0], S = tokens->dims[1];
  if (B < 1 || B > D->cfg.max_batch || S < 1) return fail(c, CG_ERR_SHAPE, "decoder: batch or length out of range");
  if (fresh) {
    CG_TRY(mixed_reset(D));
    for (int r = 0; r < B; ++r) { X.open[r] = 1; X.cur_slots.push_back(r); }
    D->B = B;
  } else if (B != D->B) return fail(c, CG_ERR_SHAPE, "decoder: append needs the cached batch size");
  Hold tk;
  CG_TRY(as_contiguous(c, tokens, &tk.t));
  const std::vector<int> rows = X.cur_slots;
  return mixed_run(D, rows, std::vector<int>((size_t)B, (int)S), (const uint32_t*)tk.t->data(), nullptr, 0, true, fresh, nullptr);
}

int mixed_truncate(cg_decoder* D, int64_t positions) {
  MixedModel& X = *D->mixed;
  if (positions == 0) return mixed_reset(D);
  for (int s : X.cur_slots) {
    if (X.pos[s] != positions && X.recurrent)
      return fail(D->c, CG_ERR_UNSUPPORTED, "decoder: a recurrent state cannot go back to an earlier position (truncate to 0 and run again)");
    if (positions < 0 || positions > X.pos[s]) return fail(D->c, CG_ERR_SHAPE, "decoder: cannot truncate to more than is cached");
  }
  for (int s : X.cur_slots) X.pos[s] = positions;
  X.tables_current = false;
  return set_state(D, 0, 0);
}

int mixed_position(cg_decoder* D, int64_t* cached) {
  MixedModel& X = *D->mixed;
  *cached = X.cur_slots.empty() ? 0 : X.pos[X.cur_slots[0]];
  return CG_OK;
}

int mixed_begin_decode(cg_decoder* D, int steps) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  for (int s : X.cur_slots)
    if (X.pos[s] + steps > D->cfg.max_seq) return fail(c, CG_ERR_SHAPE, "decoder: cache capacity exceeded");
  if (D->generated + steps > D->cfg.max_seq) return fail(c, CG_ERR_SHAPE, "decoder: token history is full");
  if (X.tables_current) return CG_OK;
  Portion p;
  p.slots = X.cur_slots;
  p.lens.assign(p.slots.size(), 1);
  for (int s : p.slots) p.pos0.push_back(X.pos[s]);
  p.M = (int64_t)p.slots.size();
  RowsDev rd;
  Chunks ch;
  CG_TRY(write_tables(D, p, X.tab_dec, &rd, &ch));
  CG_TRY(set_state(D, 0, D->generated));
  X.tables_current = true;
  return CG_OK;
}

int mixed_step(cg_decoder* D) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int R = (int)D->B;
  const int32_t* d = (const int32_t*)X.tab_dec->data();
  RowsDev rd;
  rd.slot = d; rd.start = d + R; rd.pos0 = d + 2 * R + 1; rd.tok_row = d + 3 * R + 1;
  rd.step = D->pos_dev();
  rd.rows = R;
  rd.M = R;
  CG_TRY(walk(D, rd, (const uint32_t*)D->cur->data(), nullptr, nullptr));
  CG_TRY(final_rows(D, rd.tok_row, nullptr, R, D->xl->data()));  // row i of the batch is token i
  float* lg = (float*)D->logits->data();
  CG_TRY(lin(D, D->xl->data(), X.Wp, R, D->head, 0, D->Vp, lg, D->Vp));
  return k_launch_argmax(c, lg, R, D->Vp, 1, D->cfg.final_softcap, (uint32_t*)D->cur->data(), (uint32_t*)D->history->data(),
                         D->cfg.max_seq, D->count_dev(), D->pos_dev(), 1, (unsigned long long*)D->best->data());
}

void mixed_advance(cg_decoder* D, int steps) {
  MixedModel& X = *D->mixed;
  for (int s : X.cur_slots) X.pos[s] += steps;
}

}  // namespace cg

using namespace cg;

extern "C" {

int32_t cg_decoder_seq_open(cg_decoder* D, int32_t* slot) {
  if (!D || !slot) return CG_ERR_INVALID;
  if (!D->mixed || !D->finalized) return fail(D->c, CG_ERR_UNSUPPORTED, "decoder: sequences of unequal length need a finalized layer-by-layer decoder");
  MixedModel& X = *D->mixed;
  for (size_t s = 0; s < X.open.size(); ++s)
    if (!X.open[s]) {
      X.open[s] = 1;
      X.pos[s] = 0;
      *slot = (int32_t)s;
      return CG_OK;
    }
  return fail(D->c, CG_ERR_SHAPE, "decoder: every sequence slot is taken");
}

int32_t cg_decoder_seq_close(cg_decoder* D, int32_t slot) {
  if (!D || !D->mixed) return CG_ERR_INVALID;
  MixedModel& X = *D->mixed;
  if (slot < 0 || slot >= (int32_t)X.open.size() || !X.open[slot]) return fail(D->c, CG_ERR_INVALID, "decoder: no such sequence");
  X.open[slot] = 0;
  // a closed sequence leaves the current rows; the others can no longer be decoded as one batch
  if (std::find(X.cur_slots.begin(), X.cur_slots.end(), slot) != X.cur_slots.end()) {
    X.cur_slots.clear();
    X.tables_current = false;
    D->B = 0;
  }
  return CG_OK;
}

int32_t cg_decoder_run(cg_decoder* D, int32_t rows, const int32_t* slots, const int32_t* lens, const uint32_t* tokens, int32_t n_want,
                       const int32_t* want, int32_t greedy, cg_tensor** logits_out) {
  CG_LAZY_EAGER_SCOPE(D ? D->c : nullptr);
  if (!D || rows < 1 || !slots || !lens || !tokens || n_want < 0 || (n_want && (!want || !logits_out))) return CG_ERR_INVALID;
  cg_ctx* c = D->c;
  if (!D->mixed || !D->finalized) return fail(c, CG_ERR_UNSUPPORTED, "decoder: sequences of unequal length need a finalized layer-by-layer decoder");
  int64_t n = 0;
  for (int r = 0; r < rows; ++r) {
    if (lens[r] < 1) return fail(c, CG_ERR_SHAPE, "decoder: length out of range");
    n += lens[r];
  }
  Hold tk;
  CG_TRY(cg_ndarray_from_vec_u32(c, tokens, n, &n, 1, &tk.t));
  return mixed_run(D, std::vector<int>(slots, slots + rows), std::vector<int>(lens, lens + rows), (const uint32_t*)tk.t->data(), want, n_want,
                   greedy != 0, true, logits_out);
}

int32_t cg_decoder_keep_residuals(cg_decoder* D, int32_t on) {
  if (!D || !D->mixed) return CG_ERR_INVALID;
  D->mixed->keep = on != 0;
  return CG_OK;
}

int32_t cg_decoder_residuals(cg_decoder* D, cg_tensor** out) {
  if (!D || !D->mixed || !out) return CG_ERR_INVALID;
  if (!D->mixed->kept) return fail(D->c, CG_ERR_INVALID, "decoder: no residuals were kept");
  D->mixed->kept->rc++;
  *out = D->mixed->kept;
  return CG_OK;
}

}  // extern "C"
