// mixers.h — launchers of the kernels that decoders built layer by layer use beside the GEMMs
// (decoder_mixed.cu): the residual-stream update, latent attention (latent.cu) and the linear
// recurrences with short convolutions (recurrent.cu).
//
// A batch is a set of rows of unequal length: row r brings the next tokens of the sequence in
// slot[r], packed row after row, so token m of the batch belongs to row tok_row[m].
#pragma once

#include "kernels.h"

namespace cg {

struct RowsDev {
  const int32_t* slot;     // [rows] where the row's cache and state live
  const int32_t* start;    // [rows + 1] first packed token of the row
  const int32_t* pos0;     // [rows] position of its first token when *step was 0
  const int32_t* tok_row;  // [M]
  const int64_t* step;     // decode steps taken since the tables were written
  int rows;
  int64_t M;
};

#ifdef __CUDACC__
__device__ __forceinline__ int64_t row_pos0(const RowsDev& r, int row) { return r.pos0[row] + *r.step; }
#endif

// One pass over the residual stream, row by row:
//   src  = table[tokens[m]]            (tokens set)
//        | y[m]                        (y set)
//   x[m] = (add ? x[m] : 0) + (g1 ? rms(src) * g1 : src)
//   out  = g2 ? rms(x) * g2 : x        (out set; f32 or bf16)
//   x0   = x                           (x0 set; a second copy in out's type)
// With pick set, x is read only: out[dst[m]] = rms(x[pick[m]]) * g2.
struct RowUpdate {
  const uint32_t* tokens = nullptr;
  const void* table = nullptr;
  int table_bf16 = 0;
  int64_t vocab = 0;
  const float* y = nullptr;
  int64_t ldy = 0;
  const float* g1 = nullptr;
  int add = 0;
  float* x = nullptr;
  int64_t ldx = 0;
  const float* g2 = nullptr;
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

// out[M, N] = x[M, K] w[N, K]^T in f32 (CUDA cores)
int gemm_nt_f32(cg_ctx* c, const float* x, int64_t ldx, const float* w, int64_t ldw, float* out, int64_t ldo, int64_t M, int64_t N,
                int64_t K);
// out[m, i] = act(gu[m, i]) * gu[m, F + i] in f32
int k_launch_glu_f32(cg_ctx* c, const float* gu, int64_t M, int64_t F, int act, float* out);

// Rotary tables cos, sin [T, r / 2] of angles p * base^(-2 i / r), evaluated in double precision
int k_launch_pair_rope_tables(cg_ctx* c, double base, int64_t T, int r, float* cos_t, float* sin_t);

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
  // decode scratch (bf16 path)
  float* qa = nullptr;     // [M, H, Lw] queries mapped into the cached rows' space
  float* oc = nullptr;     // [M, H, R] attention output in that space
};
int k_launch_latent_prep(cg_ctx* c, const LatentArgs& a);
int k_launch_latent_attn(cg_ctx* c, const LatentArgs& a);  // any sizes; one CTA per (token, head)

// --------------------------------------------------------- recurrences with a matrix state ----
// Both mixers: [conv segment | gate segment | small segment] = W_in h.  The conv segment passes a
// causal convolution per channel and silu and then holds, per token, queries and keys (KH heads of
// dk) and values (H heads of dv); head h uses query/key head h / (H / KH).
//   delta: S <- g S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q        (S is dk x dv)
//   ssd:   S <- g S + dt k v^T;  o = S^T q + D v
struct RecurArgs {
  int delta;
  int H, KH, dk, dv;
  int C, taps;             // conv channels
  int q_off, k_off, v_off; // columns inside the conv segment
  int gate_off, small_off; // columns inside the projection
  const float* proj;       // [M, ldp]
  int64_t ldp;
  const float* conv_w;     // [C, taps]
  const float* conv_b;     // [C] or null
  float* tail;             // [slots, taps - 1, C] last inputs of the convolution
  const float *a_log, *dt_bias;  // [H]
  const float* dskip;      // [H], ssd
  float* S;                // [slots, H, dk, dv] f32
  float* cv;               // [M, ldc] conv outputs (q, k unit vectors for delta)
  int64_t ldc;
  float *gl, *co;          // [M, H] log decay; beta (delta) or dt (ssd)
  float* o;                // [M, H * dv]
  const float* norm;       // delta: [dv]; ssd: [H * dv]
  int norm_groups;         // ssd
  float eps;
  void* att;               // [M, ld_att]
  int64_t ld_att;
  int bf16;                // element type of att
  RowsDev rows;
};
int k_launch_conv_heads(cg_ctx* c, const RecurArgs& a);   // proj -> cv, gl, co
int k_launch_conv_tail(cg_ctx* c, const RecurArgs& a);    // remembers the last inputs; after k_launch_conv_heads
int k_launch_recur_steps(cg_ctx* c, const RecurArgs& a);  // cv -> o, S: token by token, any sizes
int k_launch_gated_norm(cg_ctx* c, const RecurArgs& a);   // o -> att

}  // namespace cg
