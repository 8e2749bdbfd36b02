// decoder_mixed.cu — decoders whose layers carry different sequence mixers and may run in a loop:
// their weights, per-sequence caches and states, and the walk over their layers.  The entry points
// (prefill, append, decode with its captured graph, generate) are those of decoder.cu.
//
// A sequence lives in a slot.  Per layer run (a looped layer counts once per pass) a slot holds
//   latent attention   [max_seq, Lw] cached rows (normed latent, rotated key part)
//   delta, ssd         an f32 matrix per head and the last inputs of the convolutions
// Nothing is cleared when a slot is reused: a row whose first position is 0 starts from zeros.
// Batches are rows of unequal length, packed token after token; every kernel finds a token's row,
// slot and position through the row tables (RowsDev).  In a decode step the tables stay as they
// are and a device counter moves all positions, so the step is one CUDA graph.
//
// Fused steps: all projections of a mixer are one GEMM (w_in); a post-norm, the residual add and
// the next pre-norm are one pass (k_row_update), which also writes the two-part rows a looped
// input reads.  Matrices are padded with zeros to multiples of 8 where the tensor cores want it.

#include <algorithm>
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
  cg_tensor *n1 = nullptr, *n1b = nullptr, *n2 = nullptr, *n2b = nullptr;
  cg_tensor *w_in = nullptr, *w_o = nullptr, *w_gu = nullptr, *w_down = nullptr;
  int64_t Np = 0;       // columns of the projection
  int64_t Fp = 0;       // padded feed-forward width
  int Do = 0;           // columns a head takes in the mixer's output
  int64_t Ko = 0;       // width of the mixer's output
  // latent attention
  cg_tensor *c_gain = nullptr, *uk = nullptr, *uv = nullptr, *w_kv = nullptr, *cos_t = nullptr, *sin_t = nullptr;
  int64_t Lw = 0;       // width of a cached row
  int dkv_off = 0, Dq = 0;
  // recurrences
  cg_tensor *conv_w = nullptr, *conv_b = nullptr, *a_log = nullptr, *dt_bias = nullptr, *dskip = nullptr, *norm = nullptr;
  bool chunked = false;  // prompts run on the tensor cores, 64 tokens at a time
  int H = 0, KH = 0, dk = 0, dv = 0, dvs = 0, C = 0, gate_off = 0, small_off = 0, q_off = 0, k_off = 0, v_off = 0;
};

struct MixedRun {
  int layer;
  bool starts_pass;
  cg_tensor *cache = nullptr;                  // latent attention
  cg_tensor *state = nullptr, *tail = nullptr;  // recurrences
};

struct MixedModel {
  std::vector<MixedLayer> layers;
  std::vector<MixedRun> runs;
  bool loop = false;
  bool f32 = false;
  int64_t Wp = 0;       // padded width of the residual stream
  cg_tensor *embed_norm = nullptr, *w_loop = nullptr;
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
  CG_TRY(new2(c, ST_F32, D->cfg.max_seq, std::max<int64_t>(r / 2, 1), &L.cos_t));
  CG_TRY(new2(c, ST_F32, D->cfg.max_seq, std::max<int64_t>(r / 2, 1), &L.sin_t));
  if (r) CG_TRY(k_launch_pair_rope_tables(c, k.rot_base, D->cfg.max_seq, (int)r, (float*)L.cos_t->data(), (float*)L.sin_t->data()));
  return CG_OK;
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
    CG_TRY(norm_weight(D, mx + "norm", L.dv, &L.norm));
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
    CG_TRY(norm_weight(D, mx + "norm", inner, &L.norm));
  }
  CG_TRY(norm_weight(D, mx + "A_log", L.H, &L.a_log));
  CG_TRY(norm_weight(D, mx + "dt_bias", L.H, &L.dt_bias));
  L.Do = L.dv;
  L.Ko = up8(inner);
  CG_TRY(new2(c, st, X.Wp, L.Ko, &L.w_o));
  return place_all(D, mx + "o", W, inner, L.w_o, 0);
}

void forget_graph(cg_decoder* D) {
  if (D->graph) { cudaGraphExecDestroy(D->graph); D->graph = nullptr; }
}

int ensure_mixed(cg_decoder* D, int64_t M) {
  MixedModel& X = *D->mixed;
  if (M <= X.cap) return CG_OK;
  cg_ctx* c = D->c;
  forget_graph(D);  // it holds the old buffers
  int64_t np = 0, cc = 0, hh = 0, inner = 0, ko = 0, fp = 0, qw = 0, lw = 0, qkv = 0, kh = 0;
  for (const MixedLayer& L : X.layers) {
    np = std::max(np, L.Np);
    ko = std::max(ko, L.Ko);
    fp = std::max(fp, L.Fp);
    if (L.k.mixer == CG_MIX_LATENT) {
      qw = std::max<int64_t>(qw, (int64_t)L.k.heads * L.Dq);
      lw = std::max(lw, L.Lw);
    } else {
      cc = std::max<int64_t>(cc, up8(L.C));
      hh = std::max<int64_t>(hh, L.H);
      inner = std::max<int64_t>(inner, (int64_t)L.H * L.dvs);
      if (L.chunked) {
        qkv = std::max<int64_t>(qkv, 2 * L.KH * up16(L.dk) + (int64_t)L.H * L.dvs);
        kh = std::max<int64_t>(kh, L.KH);
      }
    }
  }
  const int st = X.act_storage();
  CG_TRY(new2(c, ST_F32, M, X.Wp, &X.x));
  CG_TRY(new2(c, st, M, X.Wp, &X.xn));
  CG_TRY(new2(c, ST_F32, M, X.Wp, &X.y));
  if (X.loop) CG_TRY(new2(c, st, M, 2 * X.Wp, &X.xcat));
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
    CG_TRY(new2(c, st, M, lw, &X.cpk));
  }
  drop(X.tok);
  CG_TRY(new_tensor(c, CG_U32, ST_U32, &M, 1, &X.tok));
  X.cap = M;
  return CG_OK;
}

// out[M, N] = x[M, K] w[row0 .. row0 + N, K]^T; out_bf16 only in a bf16 context
int lin(cg_decoder* D, const void* x, int64_t ldx, int64_t M, const cg_tensor* w, int64_t row0, int64_t N, void* out, int64_t ldo,
        bool out_bf16 = false) {
  cg_ctx* c = D->c;
  const int64_t K = w->dims[1];
  if (D->mixed->f32)
    return gemm_nt_f32(c, (const float*)x, ldx, (const float*)w->data() + row0 * K, K, (float*)out, ldo, M, N, K);
  const __nv_bfloat16* xb = (const __nv_bfloat16*)x;
  const __nv_bfloat16* wb = (const __nv_bfloat16*)w->data() + row0 * K;
  if (gemm_dec_supported(M, K)) {
    DecGemm g;
    g.x = xb; g.ldx = ldx; g.w = wb; g.ldw = K; g.w_rows = N;
    g.out = out; g.ldo = ldo; g.residual = nullptr; g.out_mode = out_bf16 ? 1 : 0;
    g.push = nullptr; g.dual = 0; g.act = 0;
    g.M = M; g.N = N; g.K = K;
    return gemm_dec(c, g);
  }
  const int splits = gemm_tc_pick_splits(M, N, K);
  float* ws = (int64_t)splits * M * N <= D->splitk_floats ? (float*)D->splitk->data() : nullptr;
  return gemm_tc(c, xb, ldx, wb, K, out, ldo, nullptr, M, N, K, out_bf16 ? 1 : 0, splits, ws);
}

// hact = act(x gate^T) * (x up^T)
int glu(cg_decoder* D, const MixedLayer& L, const void* x, int64_t M) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int64_t K = X.Wp, F = L.Fp;
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
    CG_TRY(lin(D, X.cpk->data(), L.Lw, rd.M, L.w_kv, 0, kvw, kv, kvw, true));
  } else {
    int64_t at = 0;
    for (int r = 0; r < R; ++r) {
      const int64_t n = p->pos0[r] + p->lens[r];
      CG_TRY(lin(D, (const char*)a.cache + (size_t)p->slots[r] * a.Tmax * L.Lw * es, L.Lw, n, L.w_kv, 0, kvw, kv + (size_t)at * kvw * es, kvw,
                 true));
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
  a->delta = L.k.mixer == CG_MIX_DELTA ? 1 : 0;
  a->H = L.H; a->KH = L.KH; a->dk = L.dk; a->dv = L.dv; a->dvs = L.dvs; a->C = L.C; a->taps = L.k.conv;
  a->q_off = L.q_off; a->k_off = L.k_off; a->v_off = L.v_off;
  a->conv_w = (const float*)L.conv_w->data();
  a->conv_b = L.conv_b ? (const float*)L.conv_b->data() : nullptr;
  a->tail = (float*)run.tail->data();
  a->a_log = (const float*)L.a_log->data(); a->dt_bias = (const float*)L.dt_bias->data();
  a->dskip = L.dskip ? (const float*)L.dskip->data() : nullptr;
  a->S = (float*)run.state->data();
  a->gl = (float*)X.gl->data(); a->co = (float*)X.co->data();
  a->o = (float*)X.ro->data();
  a->rows = rd;
}

// One token per row: one kernel.  Prompts in a bf16 context: chunks on the tensor cores, on bf16
// projections (the gates' projections stay f32).  Otherwise token by token.
int recurrent_layer(cg_decoder* D, const MixedLayer& L, MixedRun& run, const RowsDev& rd, const Portion* p, const Chunks* ch) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int64_t M = rd.M, K = X.Wp;
  GatedNorm n;
  n.delta = L.k.mixer == CG_MIX_DELTA ? 1 : 0;
  n.H = L.H; n.dv = L.dv; n.dvs = L.dvs; n.norm_groups = L.k.norm_groups;
  n.o = (const float*)X.ro->data();
  n.norm = (const float*)L.norm->data(); n.eps = D->cfg.rms_eps;
  n.att = X.att->data(); n.ld_att = L.Ko; n.att_bf16 = X.f32 ? 0 : 1;
  n.M = M;
  if (L.chunked && p && p->max_len >= 8) {
    ChunkArgs a;
    recurrent_base(D, L, run, rd, &a);
    __nv_bfloat16* pb = (__nv_bfloat16*)X.proj->data();
    float* small = (float*)(pb + M * L.small_off);  // both fit where the f32 projection would
    const int64_t ns = L.Np - L.small_off;
    CG_TRY(lin(D, X.xn->data(), K, M, L.w_in, 0, L.small_off, pb, L.small_off, true));
    CG_TRY(lin(D, X.xn->data(), K, M, L.w_in, L.small_off, ns, small, ns));
    a.proj = pb; a.ldp = L.small_off;
    a.small = small; a.ld_small = ns;
    a.DKp = (int)up16(L.dk); a.dvp = L.dvs;
    a.q = (__nv_bfloat16*)X.qkv->data();
    a.k = a.q + M * L.KH * a.DKp;
    a.v = a.k + M * L.KH * a.DKp;
    a.rq = (float*)X.rn->data();
    a.rk = a.rq + M * L.KH;
    a.chunk_tok = ch->tok; a.chunk_len = ch->len; a.row_chunk = ch->row_chunk; a.n_chunks = ch->n;
    a.T = nullptr;
    if (a.delta) {
      CG_TRY(grow(c, ST_BF16, (int64_t)ch->n * L.H * 2 * RECUR_CHUNK * RECUR_CHUNK, &X.tinv, &X.tinv_n));
      a.T = (__nv_bfloat16*)X.tinv->data();
    }
    CG_TRY(k_launch_chunk_recurrence(c, a));
    n.gate = pb + L.gate_off; n.ldg = L.small_off; n.gate_bf16 = 1;
    return k_launch_gated_norm(c, n);
  }
  RecurArgs a;
  recurrent_base(D, L, run, rd, &a);
  CG_TRY(lin(D, X.xn->data(), K, M, L.w_in, 0, L.Np, X.proj->data(), L.Np));
  a.proj = (const float*)X.proj->data(); a.ldp = L.Np;
  a.gate_off = L.gate_off; a.small_off = L.small_off;
  a.cv = (float*)X.cv->data(); a.ldc = up8(L.C);
  n.gate = a.proj + L.gate_off; n.ldg = L.Np; n.gate_bf16 = 0;
  if ((!p || p->max_len == 1) && recur_decode_supported(L.dk, L.dv)) return k_launch_recur_decode(c, a, n);
  CG_TRY(k_launch_recur_steps(c, a));
  return k_launch_gated_norm(c, n);
}

// Embedding and all layer runs of one batch; x holds the residual stream afterwards.  p is null in
// decode steps (one token per row).
int walk(cg_decoder* D, const RowsDev& rd, const uint32_t* tokens, const Portion* p, const Chunks* ch) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int64_t M = rd.M, W = D->H, Wp = X.Wp;
  const int bf = X.f32 ? 0 : 1;
  char* cat_lo = X.loop ? (char*)X.xcat->data() : nullptr;
  char* cat_hi = X.loop ? cat_lo + (size_t)Wp * storage_bytes(X.act_storage()) : nullptr;
  const size_t nruns = X.runs.size();
  // what the row update leaves for run i: its normed input, or the first half of a pass's input rows
  auto hand_on = [&](RowUpdate& u, size_t i) {
    if (i >= nruns) return;
    if (X.runs[i].starts_pass) { u.out = cat_lo; u.ldo = 2 * Wp; u.g2 = nullptr; }
    else { u.out = X.xn->data(); u.ldo = Wp; u.g2 = (const float*)X.layers[X.runs[i].layer].n1->data(); }
  };
  RowUpdate base;
  base.x = (float*)X.x->data(); base.ldx = Wp; base.eps = D->cfg.rms_eps; base.W = (int)W;
  {
    RowUpdate u = base;
    u.tokens = tokens; u.table = D->embed->data(); u.table_bf16 = D->embed->storage == ST_BF16; u.vocab = D->cfg.vocab;
    u.g1 = (const float*)X.embed_norm->data();
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
      u.out = X.xn->data(); u.ldo = Wp; u.g2 = (const float*)L.n1->data();
      CG_TRY(k_launch_row_update(c, u, M, bf));
    }
    if (L.k.mixer == CG_MIX_LATENT) CG_TRY(latent_layer(D, L, run, rd, p));
    else CG_TRY(recurrent_layer(D, L, run, rd, p, ch));
    CG_TRY(lin(D, X.att->data(), L.Ko, M, L.w_o, 0, Wp, X.y->data(), Wp));
    RowUpdate u = base;
    u.y = (const float*)X.y->data(); u.ldy = Wp; u.add = 1;
    u.g1 = (const float*)L.n1b->data();
    if (L.k.ffn) {
      u.out = X.xn->data(); u.ldo = Wp; u.g2 = (const float*)L.n2->data();
      CG_TRY(k_launch_row_update(c, u, M, bf));
      CG_TRY(glu(D, L, X.xn->data(), M));
      CG_TRY(lin(D, X.hact->data(), L.Fp, M, L.w_down, 0, Wp, X.y->data(), Wp));
      u.g1 = (const float*)L.n2b->data();
      u.out = nullptr; u.g2 = nullptr;
    }
    hand_on(u, i + 1);
    CG_TRY(k_launch_row_update(c, u, M, bf));
    if (X.keep && p) {
      if (i == 0) {
        drop(X.kept);
        int64_t d3[3] = {(int64_t)nruns, M, W};
        CG_TRY(new_tensor(c, CG_F32, ST_F32, d3, 3, &X.kept));
      }
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
  X->layers.resize(n_layers);
  for (int i = 0; i < n_layers; ++i) {
    const cg_layer_config& k = layers[i];
    X->layers[i].k = k;
    if (k.heads < 1 || k.vdim < 1 || k.ffn < 0) return bad_size(D, i, "sizes must be positive");
    if (k.mixer == CG_MIX_LATENT) {
      if (k.dim < 1 || k.rot_dim < 0 || k.rot_dim % 2 || k.kv_rank < 1 || (k.rot_dim && !(k.rot_base > 0)))
        return bad_size(D, i, "latent attention sizes");
    } else if (k.mixer == CG_MIX_DELTA) {
      if (k.dim < 1 || k.kv_heads < 1 || k.heads % k.kv_heads || k.conv < 1) return bad_size(D, i, "delta rule sizes");
    } else if (k.mixer == CG_MIX_SSD) {
      if (k.state < 1 || k.groups < 1 || k.heads % k.groups || k.norm_groups < 1 || (k.heads * k.vdim) % k.norm_groups || k.conv < 1)
        return bad_size(D, i, "state space sizes");
    } else return bad_size(D, i, "unknown mixer");
  }
  const bool looped = loop && loop->times > 0 && loop->stop > loop->start;
  if (looped && (loop->start < 0 || loop->stop > n_layers)) return fail(D->c, CG_ERR_INVALID, "decoder: loop out of range");
  X->loop = looped;
  auto add = [&](int i, bool starts) {
    MixedRun r;
    r.layer = i;
    r.starts_pass = starts;
    X->runs.push_back(r);
  };
  const int a = looped ? loop->start : n_layers, b = looped ? loop->stop : n_layers;
  for (int i = 0; i < a; ++i) add(i, false);
  for (int t = 0; looped && t < loop->times; ++t)
    for (int i = a; i < b; ++i) add(i, i == a);
  for (int i = b; i < n_layers; ++i) add(i, false);
  X->open.assign(D->cfg.max_batch, 0);
  X->pos.assign(D->cfg.max_batch, 0);
  return CG_OK;
}

void mixed_destroy(cg_decoder* D) {
  MixedModel* X = D->mixed;
  if (!X) return;
  for (MixedLayer& L : X->layers)
    for (cg_tensor** t : {&L.n1, &L.n1b, &L.n2, &L.n2b, &L.w_in, &L.w_o, &L.w_gu, &L.w_down, &L.c_gain, &L.uk, &L.uv, &L.w_kv, &L.cos_t,
                          &L.sin_t, &L.conv_w, &L.conv_b, &L.a_log, &L.dt_bias, &L.dskip, &L.norm})
      drop(*t);
  for (MixedRun& r : X->runs) { drop(r.cache); drop(r.state); drop(r.tail); }
  for (cg_tensor** t : {&X->embed_norm, &X->w_loop, &X->tab_run, &X->tab_dec, &X->x, &X->xn, &X->xcat, &X->y, &X->proj, &X->cv, &X->gl,
                        &X->co, &X->ro, &X->att, &X->hact, &X->gu, &X->q, &X->cpk, &X->tok, &X->xw, &X->kept, &X->qkv, &X->rn,
                        &X->tinv, &X->kv, &X->lat})
    drop(*t);
  delete X;
  D->mixed = nullptr;
}

int mixed_finalize(cg_decoder* D) {
  cg_ctx* c = D->c;
  MixedModel& X = *D->mixed;
  const int64_t W = D->H;
  const int st = X.act_storage();
  for (size_t i = 0; i < X.layers.size(); ++i) {
    MixedLayer& L = X.layers[i];
    const std::string l = "l" + std::to_string(i) + ".";
    CG_TRY(norm_weight(D, l + "norm1", W, &L.n1));
    CG_TRY(norm_weight(D, l + "norm1b", W, &L.n1b));
    if (L.k.mixer == CG_MIX_LATENT) CG_TRY(finalize_latent(D, L, l + "mix."));
    else CG_TRY(finalize_recurrent(D, L, l + "mix."));
    if (L.k.ffn) {
      const int64_t F = L.k.ffn;
      L.Fp = up8(F);
      CG_TRY(norm_weight(D, l + "norm2", W, &L.n2));
      CG_TRY(norm_weight(D, l + "norm2b", W, &L.n2b));
      CG_TRY(new2(c, st, 2 * L.Fp, X.Wp, &L.w_gu));
      CG_TRY(place_all(D, l + "mlp.gate", F, W, L.w_gu, 0));
      CG_TRY(place_all(D, l + "mlp.up", F, W, L.w_gu, L.Fp));
      CG_TRY(new2(c, st, X.Wp, L.Fp, &L.w_down));
      CG_TRY(place_all(D, l + "mlp.down", W, F, L.w_down, 0));
    }
    // the originals of this layer are no longer needed
    for (auto it = D->params.begin(); it != D->params.end();) {
      if (it->first.compare(0, l.size(), l) == 0) { release(it->second); it = D->params.erase(it); }
      else ++it;
    }
  }
  const int64_t slots = D->cfg.max_batch;
  for (MixedRun& r : X.runs) {
    const MixedLayer& L = X.layers[r.layer];
    if (L.k.mixer == CG_MIX_LATENT) {
      CG_TRY(new2(c, st, slots * D->cfg.max_seq, L.Lw, &r.cache));
    } else {
      CG_TRY(new2(c, ST_F32, slots * L.H * L.dk, L.dvs, &r.state));
      CG_TRY(new2(c, ST_F32, slots * L.k.conv, L.C, &r.tail));
    }
  }
  if (X.loop) {
    CG_TRY(new2(c, st, X.Wp, 2 * X.Wp, &X.w_loop));
    CG_TRY(place(D, "loop.in", W, 2 * W, 0, W, 0, W, X.w_loop, 0, 0));
    CG_TRY(place(D, "loop.in", W, 2 * W, 0, W, W, W, X.w_loop, 0, X.Wp));
  }
  CG_TRY(norm_weight(D, "embed.norm", W, &X.embed_norm));
  CG_TRY(norm_weight(D, "final.norm", W, &D->ln_f));
  CG_TRY(new2(c, st, D->cfg.vocab, W, &D->embed, false));
  CG_TRY(place_all(D, "embed", D->cfg.vocab, W, D->embed, 0));
  CG_TRY(new2(c, st, D->cfg.vocab, X.Wp, &D->head));
  CG_TRY(place_all(D, "head", D->cfg.vocab, W, D->head, 0));
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
  for (const MixedLayer& L : X.layers) widest = std::max({widest, L.Np, 2 * L.Fp});
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
      RowUpdate u;
      u.x = (float*)X.x->data(); u.ldx = X.Wp; u.eps = D->cfg.rms_eps; u.W = (int)D->H;
      u.pick = pd; u.dst = pd + np;
      u.out = X.xw->data(); u.ldo = X.Wp; u.g2 = (const float*)D->ln_f->data();
      CG_TRY(k_launch_row_update(c, u, (int64_t)np, X.f32 ? 0 : 1));
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
  for (int s : X.cur_slots)
    if (X.pos[s] != positions)
      return fail(D->c, CG_ERR_UNSUPPORTED, "decoder: a recurrent state cannot go back to an earlier position (truncate to 0 and run again)");
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
  RowUpdate u;
  u.x = (float*)X.x->data(); u.ldx = X.Wp; u.eps = D->cfg.rms_eps; u.W = (int)D->H;
  u.pick = rd.tok_row;  // row i of the batch is token i
  u.out = D->xl->data(); u.ldo = X.Wp; u.g2 = (const float*)D->ln_f->data();
  CG_TRY(k_launch_row_update(c, u, R, X.f32 ? 0 : 1));
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
