// mixers.h — launchers of the kernels that decoders built layer by layer use beside the GEMMs
// (decoder_mixed.cu): the residual-stream update, latent attention (latent.cu) and the linear
// recurrences with short convolutions (recurrent.cu).
// Batches are rows of unequal length (RowsDev, kernels.h).
#pragma once

#include "kernels.h"

namespace cg {

// One pass over the residual stream, row by row:
//   src  = scale * table[tokens[m]]    (tokens set)
//        | y[m] (y set) + sum over the token's experts i of wts[m top + i] ye[pos[m top + i]] (top > 0;
//          wts null: ones)
//   x[m] = (add ? x[m] : 0) + (g1 ? norm(src) * g1 + b1 : src)
//   out  = g2 ? norm(x) * g2 + b2 : x  (out set; f32 or bf16)
//   x0   = x                           (x0 set; a second copy in out's type)
// norm divides by the root mean square, with centred after taking the mean off; biases may be null.
// With pick set, x is read only: out[dst[m]] = norm(x[pick[m]]) * g2 + b2.
struct RowUpdate {
  const uint32_t* tokens = nullptr;
  const void* table = nullptr;
  int table_bf16 = 0;
  int64_t vocab = 0;
  float scale = 1.f;
  const float* y = nullptr;
  int64_t ldy = 0;
  const float* ye = nullptr;
  int64_t ldye = 0;
  const int32_t* pos = nullptr;
  const float* wts = nullptr;
  int top = 0;
  int centred = 0;
  const float *g1 = nullptr, *b1 = nullptr;
  int add = 0;
  float* x = nullptr;
  int64_t ldx = 0;
  const float *g2 = nullptr, *b2 = nullptr;
  void* out = nullptr;
  int64_t ldo = 0;
  void* x0 = nullptr;
  int64_t ld0 = 0;
  const int32_t* pick = nullptr;
  const int32_t* dst = nullptr;
  float eps = 0.f;
  int W = 0;  // row length; columns up to the next multiple of 8 are kept zero
};
int k_launch_row_update(cg_ctx* c, const RowUpdate& u, int64_t M, int out_bf16);

// The same for hyper-connected models, whose residual stream is ns rows per token: x is [M, ns, ldx].
//   y    = y[m] | sum over the token's experts i of wts[m top + i] y[pos[m top + i]]   (top > 0)
//   x[t] = sum over s of mix[s, t] x[s] + out_w[t] y
// or, with tokens set, every x[t] = scale * table[tokens[m]].  Then
//   h    = sum over s of in_w[s] x[s]                (in_w null: all ones)
//   out  = rms(h) * g                                (out set)
//   sum[m] = sum over s of x[s]                      (sum set)
// With pick set, x is read only: out[dst[m]] = rms(sum of x[pick[m]]) * g.
// A plain residual stream is ns = 1 with mix = out_w = in_w = 1.
constexpr int MAX_STREAMS = 16;
struct StreamUpdate {
  const uint32_t* tokens = nullptr;
  const void* table = nullptr;
  int table_bf16 = 0;
  int64_t vocab = 0;
  float scale = 1.f;
  const float* y = nullptr;
  int64_t ldy = 0;
  const int32_t* pos = nullptr;
  const float* wts = nullptr;
  int top = 0;
  int ns = 1;
  const float *mix = nullptr, *out_w = nullptr, *in_w = nullptr;
  float* x = nullptr;
  int64_t ldx = 0;
  const float* g = nullptr;
  void* out = nullptr;
  int64_t ldo = 0;
  float* sum = nullptr;
  int64_t ld_sum = 0;
  const int32_t* pick = nullptr;
  const int32_t* dst = nullptr;
  float eps = 0.f;
  int W = 0;  // row length; columns up to the next multiple of 8 are kept zero
};
int k_launch_stream_update(cg_ctx* c, const StreamUpdate& u, int64_t M, int out_bf16);

// ---------------------------------------------- sublayers side by side, averages over depth ----
// x[m] += y[m] + y_bias + rms(normed0[m]) * gain0 + rms(normed1[m]) * gain1
//         + sum over the token's experts i of wts[m top + i] ye[pos[m top + i]]
// (y, y_bias and the normed pair may be null), and a copy of the result in the GEMMs' type.
struct BranchSum {
  float* x = nullptr;
  int64_t ldx = 0;
  const float *y = nullptr, *y_bias = nullptr;
  int64_t ldy = 0;           // of y, the normed pair and ye
  const float* normed[2] = {nullptr, nullptr};
  const float* gain[2] = {nullptr, nullptr};
  const float* ye = nullptr;
  const int32_t* pos = nullptr;
  const float* wts = nullptr;
  int top = 0;
  void* copy = nullptr;
  int64_t ld_copy = 0;
  float eps = 0.f;
  int W = 0;                 // row length; columns up to the next multiple of 8 are zero
};
int k_launch_branch_sum(cg_ctx* c, const BranchSum& u, int64_t M, int bf16);

// v = scale * table[tokens[m]] (tokens set) or x[m] + rms(y[m]) * y_gain (y may be null: x[m]);
// depth[n][m] = v;  x[m] = sum over j < n of average[j] depth[j][m] + average[n] v (average null: v);
// out = rms(x[m]) * g (out set);  kept[m] = x[m] (kept set).
struct DepthUpdate {
  const uint32_t* tokens = nullptr;
  const void* table = nullptr;
  int table_bf16 = 0;
  int64_t vocab = 0;
  float scale = 1.f;
  float* x = nullptr;
  int64_t ldx = 0;           // of x and depth
  const float *y = nullptr, *y_gain = nullptr;
  int64_t ldy = 0;
  float* depth = nullptr;
  int64_t depth_stride = 0;
  const float* average = nullptr;
  int n = 0;
  const float* g = nullptr;
  void* out = nullptr;
  int64_t ldo = 0;
  float* kept = nullptr;
  int64_t ld_kept = 0;
  float eps = 0.f;
  int W = 0;
};
int k_launch_depth_update(cg_ctx* c, const DepthUpdate& u, int64_t M, int bf16);

// out[m, j] = gelu(z[m, j]) * table[tokens[m], off + j] for j < n, 0 for n <= j < ldo
struct TokenGate {
  const uint32_t* tokens;
  int64_t vocab;
  const void* table;         // in the type of out
  int64_t ld_table, off;
  const float* z;
  int64_t ldz;
  int n;
  void* out;
  int64_t ldo;
};
int k_launch_token_gate(cg_ctx* c, const TokenGate& a, int64_t M, int bf16);
// out[m, n] = gelu(x[m, n] + bias[n]) in f32 (out may be x)
int k_launch_bias_gelu_f32(cg_ctx* c, const float* x, int64_t ldx, const float* bias, int64_t M, int64_t N, float* out, int64_t ldo);

// ------------------------------------------------------------- gated diagonal recurrence ----
// See lru.cu.  W channels in `blocks` equal blocks; the state and the convolution's last inputs (kept by
// position modulo taps) are f32.
struct LruArgs {
  const void *y, *x;         // [M, ldx] columns of the projection, without their biases
  int64_t ldx;
  int in_bf16;               // their type; decode steps take f32
  const float *yb, *xb;      // [W]
  int W, blocks, taps;
  const float *conv_w, *conv_b;  // [W, taps], [W]
  const void *ra, *ri;       // [W, W / blocks] in the type of u and out
  const float *ra_b, *ri_b, *f;  // [W]; f = -8 softplus(lam)
  float *S, *tail;           // [slots, W], [slots, taps, W]
  void* u;                   // [M, W] scratch, prompts
  float *a, *b;              // [M, W] scratch, prompts
  const int32_t *chunk_tok, *chunk_len;  // [n_chunks] first packed token, tokens (prompts)
  int n_chunks;
  void* out;
  int64_t ld_out;
  int out_bf16;
  RowsDev rows;
};
int k_launch_lru_prompt(cg_ctx* c, const LruArgs& a);
int k_launch_lru_decode(cg_ctx* c, const LruArgs& a);

// x[i] = x[i] * f + v
int k_launch_affine(cg_ctx* c, float* x, int64_t n, float f, float v);
// x[i] = max(x[i], 0)^2 in f32
int k_launch_relu2_f32(cg_ctx* c, float* x, int64_t n);

// out[m, i] = act(gu[m, i]) * gu[m, F + i] in f32
int k_launch_glu_f32(cg_ctx* c, const float* gu, int64_t M, int64_t F, int act, float* out);

// Rotary tables cos, sin [T, r / 2] of angles p * f_i, f_i = base^(-2 i / r), evaluated in double precision.
// factor > 0 stretches the slow pairs (Llama 3.1): with l = 2 pi / f, f stays where l < original / high,
// becomes f / factor where l > original / low, and a blend of both in between.
struct PairRope {
  double base = 0, factor = 0, low = 0, high = 0, original = 0;
};
int k_launch_pair_rope_tables(cg_ctx* c, const PairRope& f, int64_t T, int r, float* cos_t, float* sin_t);

// ------------------------------------------------------------- attention over a row batch ----
// Grouped-query attention with per-layer sizes, window and sink on rows of unequal length.  Heads take
// Dk (queries, keys) and Dv (values) columns in the projection, the cache and the output, of which d
// and dv are real and the rest zero.
struct RowsAttnArgs {
  const float* proj;       // [M, ldp]: H query heads, G key heads, G value heads
  int64_t ldp;
  int H, G, d, dv, Dk, Dv;
  const float *q_gain, *k_gain;  // [H Dk], [G Dk]: norms over all query / key heads at once; null: none
  int head_norm = 0;       // norms per head, without gains
  float eps, scale;
  int rot;                 // rotated components, neighbouring pairs
  const float *cos_t, *sin_t;    // [Tmax, rot / 2]
  int64_t window;          // 0 = none
  int64_t keep_first = 0;  // with a window: these first positions stay visible
  const float* sink;       // [H] or null
  float out_scale = 1.f;   // head h of token m is multiplied by out_scale and, with a gate, by
  const float* gate = nullptr;  // sigmoid(gate[m * ldp + h]), with wide_gate value e of it by sigmoid(gate[m * ldp + h * Dv + e])
  int wide_gate = 0;
  const float* q_temp = nullptr;  // [Tmax] factor on the query at a position
  const float* bias = nullptr;  // bias[h * ld_bias + distance] is taken off the scores
  int64_t ld_bias = 0;
  void* q;                 // [M, H Dk]
  void *k_cache, *v_cache; // [slots, G, Tmax, Dk | Dv]
  int64_t Tmax, slots;
  void* att;               // [M, ld_att], head h at column h * Dv
  int64_t ld_att;
  int bf16;                // element type of q, the cache and att
  RowsDev rows;
};
int k_launch_rows_qkv(cg_ctx* c, const RowsAttnArgs& a);   // norms, rotation, q, cache append
int k_launch_rows_attn(cg_ctx* c, const RowsAttnArgs& a);  // any sizes; one CTA per (token, head)

// ------------------------------------------------------------------ latent attention ----
// A cached row is [c (R values), rotated key part (r), zeros up to Lw].  Per head the key is
// [Wuk c, rotated part] and the value Wuv c.
struct LatentArgs {
  const float* proj;       // [M, ldp]: q (H heads of d + r), then at column dkv_off the R + r rows of the down projection
  int64_t ldp;
  int dkv_off;
  int H, d, r, dv, R;
  float scale, eps;
  const float *cos_t, *sin_t;  // [Tmax, r / 2]
  const float* c_gain;     // [R]
  void* cache;             // [slots, Tmax, Lw]
  int64_t Lw, Tmax;
  void* q_out;             // [M, H * Dq]: [unrotated d, rotated r, zeros]
  int Dq;
  void* c_out;             // [M, Lw] packed copy of the new cache rows, or null
  const void *uk, *uv;     // [H * d, R], [H * dv, R]
  void* att;               // [M, ld_att], head h at column h * Do
  int64_t ld_att;
  int Do;
  int bf16;                // element type of cache, q_out, c_out, uk, uv, att
  RowsDev rows;
};
int k_launch_latent_prep(cg_ctx* c, const LatentArgs& a);
int k_launch_latent_attn(cg_ctx* c, const LatentArgs& a);  // any sizes; one CTA per (token, head)

// A few new tokens per row in a bf16 context: queries are mapped into the cached rows' space, so
// that all heads attend over the same cached rows (read once), and the result is mapped back.
// Includes what k_launch_latent_prep does, without q_out.
constexpr int LATENT_DECODE_TOKENS = 64;
bool latent_decode_supported(int d, int R, int64_t Lw);
size_t latent_decode_scratch(const LatentArgs& a, int64_t M);  // bytes
int k_launch_latent_decode(cg_ctx* c, const LatentArgs& a, void* scratch);

// --------------------------------------------------------- recurrences with a matrix state ----
// [conv segment | gate segment | small segment] = W_in h.  The conv segment passes a causal
// convolution per channel (taps 0: none) and silu (without `linear`) and then holds, per token, queries and keys (KH heads
// of dk) and values (H heads of dv), the heads qs and vs columns apart; head h uses query/key head
// h / (H / KH).
//   delta:     S <- g S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q        (S is dk x dv)
//   ssd:       S <- g S + dt k v^T;  o = S^T q + D v
//   lightning: S <- g S + k v^T;  o = S^T q, g a constant per head (log_decay set), no convolution
// With key_decay g is a number per head and key channel, on the rows of S, from a low-rank projection:
//   z = W_a2 (W_a1 h),  ln g = -coef softplus(sign (z + z_bias)),  heads zs columns apart in z
// (lightning's form with key_decay is gated linear attention, linear and with q times q_scale).
// The convolution's last inputs are kept by position modulo taps, so that in a decode step blocks
// may read old inputs while another block writes the new one.
struct RecurBase {
  int delta;
  int H, KH, dk, dv, dvs;  // dvs: dv rounded up to a multiple of 8, the row length of S and o
  int qs, vs;              // columns from one head to the next in the conv segment
  int C, taps;             // conv channels
  int q_off, k_off, v_off; // columns inside the conv segment
  const float* conv_w;     // [C, taps]
  const float* conv_b;     // [C] or null
  float* tail;             // [slots, taps, C]
  const float *a_log, *dt_bias;  // [H]
  int linear = 0;
  float q_scale = 1.f;     // on queries that are not made unit vectors
  int key_decay = 0, zs = 0;
  const float *coef = nullptr, *z_bias = nullptr;  // [H], [H zs]
  float z_sign = 1.f;
  const float* log_decay = nullptr;  // [H], lightning
  const float* dskip;      // [H], ssd; null: none
  float* S;                // [slots, H, dk, dvs] f32
  float *gl, *co;          // [M, H] log decay (key_decay: [M, H zs]); beta (delta) or dt (ssd)
  float* o;                // [M, H * dvs]
  RowsDev rows;
};
// Token by token, any sizes and row lengths, f32.
struct RecurArgs : RecurBase {
  const float* proj;       // [M, ldp]
  int64_t ldp;
  int gate_off, small_off; // columns inside the projection
  float* cv;               // [M, ldc] conv outputs (q, k unit vectors for delta)
  int64_t ldc;
  // low-rank projections: columns of W_a1 h and W_g1 h inside the projection, and the second factors
  // [H zs, a_rank] and [H dv, g_rank] (f32 or bf16); w_g2 null: the gate is a segment of the projection
  int a1_off = 0, g1_off = 0, a_rank = 0, g_rank = 0, w_bf16 = 0;
  const void *w_a2 = nullptr, *w_g2 = nullptr;
  int w_staged = 0;        // set by the launcher: a decode block keeps its rows of them in shared memory
};
// out[m, n] = sum over j of x[m, j] w[n, j] in f32, for the few columns of a low-rank projection; with coef
// the log decay -coef[n / zs] softplus(sign (that + bias[n]))
struct LowRank {
  const float* x;          // [M, ldx], R columns
  int64_t ldx;
  const void* w;           // [N, R] f32 or bf16
  int w_bf16, N, R;
  const float *coef = nullptr, *bias = nullptr;
  int zs = 1;
  float sign = 1.f;
  float* out;              // [M, N]
};
int k_launch_low_rank(cg_ctx* c, const LowRank& a, int64_t M);
int k_launch_recur_steps(cg_ctx* c, const RecurArgs& a);

// Prompts, 64 tokens at a time on the tensor cores (bf16 context, dk <= 128).
constexpr int RECUR_CHUNK = 64;
struct ChunkArgs : RecurBase {
  const __nv_bfloat16* proj;  // [M, ldp]: conv segment first
  int64_t ldp;
  const float* small;      // [M, ld_small]: delta beta and a, ssd dt
  int64_t ld_small;
  int DKp, dvp;            // dk rounded up to 16, dv rounded up to 8
  __nv_bfloat16 *q, *k;    // [M, KH * DKp] conv outputs; lightning: the projections after silu
  __nv_bfloat16* v;        // [M, H * dvp]
  int64_t ldq, ldv;        // from one token to the next in q and k, and in v
  float *rq, *rk;          // [M, KH] factors that make unit vectors of them (not lightning)
  __nv_bfloat16* T;        // [chunks, H, 2, 64, 64] scratch (delta); key_decay: [chunks, H, channel_scratch]
  float* decayed = nullptr;  // key_decay: [chunks, H, dk up to 64 or 128]
  const int32_t *chunk_tok, *chunk_len;  // [n_chunks] first packed token, tokens
  const int32_t* row_chunk;              // [rows + 1]
  int n_chunks;
};
bool chunk_supported(int dk);
// key_decay (channel_chunk.cu): gl holds z; queries and keys lie DKp = up16(dk) columns apart, values dvp
int64_t channel_scratch(int dk, int delta);  // bf16 values per (chunk, head)
int k_launch_channel_chunks(cg_ctx* c, const ChunkArgs& a);
int k_launch_chunk_recurrence(cg_ctx* c, const ChunkArgs& a);

// Over each of `groups` equal parts of the H * dv values: rms, gain and times act(gate), the gate before
// the rms with gate_first, else after the gain.  delta and gated linear attention: a group per head and the
// same gains for all of them; ssd: the gate first; lightning: one group and a sigmoid.
struct GatedNorm {
  int H, dv, dvs, groups;
  int shared_gain;         // norm holds one group's gains
  int gate_first, sigmoid; // act is silu, or the sigmoid
  const float* o;          // [M, H * dvs]
  const void* gate;        // [M, ldg], H * dv columns
  int64_t ldg;
  int gate_bf16;
  const float* norm;       // [H * dv], shared_gain: [H * dv / groups]
  float eps;
  void* att;               // [M, ld_att]
  int64_t ld_att;
  int att_bf16;
  int64_t M;
};
int k_launch_gated_norm(cg_ctx* c, const GatedNorm& a);

// One new token per row: convolution, gates (their low-rank projections too), state update, read-out and,
// where its groups are the heads, the gated norm in one kernel; n gives the output.  dk, dv <= 128.
bool recur_decode_supported(int dk, int dv);
int k_launch_recur_decode(cg_ctx* c, const RecurArgs& a, const GatedNorm& n);

}  // namespace cg
