// recurrent_chunk.cu — prompts through the matrix-state recurrences, 64 tokens at a time on the
// tensor cores.
//
// With G_t the running sum of the log decays inside a chunk, S0 the state before it and u_t what
// token t writes, both recurrences read
//   S_t = e^{G_t} S0 + sum_{s<=t} e^{G_t - G_s} k_s u_s^T,      o_t = S_t^T q_t
// For the state space u_t = dt_t v_t, for lightning attention u_t = v_t and the decays are constants.  For the delta rule u solves a unit lower triangular system:
//   (I + A) U = R,  A_ts = b_t e^{G_t - G_s} (k_t . k_s) (s < t),  R_t = b_t (v_t - e^{G_t} S0^T k_t)
// T = (I + A)^-1 depends on keys and gates only, so k_delta_solve makes it for all chunks at once;
// k_delta_scan / k_ssd_scan then walk the chunks of one (row, head, 64 value columns) with S in registers.
//
// Precision.  The conv outputs are bf16 (and exact as such); unit norms are kept apart as f32 factors
// per token and head, so every product of q, k, v with itself is exact in the operands.  State,
// decays, R, U and T are f32: as a tensor-core operand each is split into a bf16 head and a bf16
// remainder (two or three products, about 16 bits), accumulation is f32, the state itself stays in
// f32 accumulators and is never rounded.
#include <algorithm>

#include "chunk_common.cuh"
#include "mixers.h"

namespace cg {

namespace {

__device__ __forceinline__ float silu(float x) { return __fdividef(x, 1.f + __expf(-x)); }  // rounded to bf16 at once
__device__ __forceinline__ float softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// ------------------------------------------------------------- short convolutions ----
// Any sizes: one block per token, a warp per query / key head or 128 other channels.  Queries and
// keys are laid out with DKp values per head, values with dvp.
__global__ void __launch_bounds__(256) k_conv_chunk_any(ChunkArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int64_t m = blockIdx.x;
  const int row = a.rows.tok_row[m];
  const int64_t p0 = row_pos0(a.rows, row);
  const int i = (int)(m - a.rows.start[row]);
  const float* tail = a.tail + (int64_t)a.rows.slot[row] * a.taps * a.C;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  auto conv = [&](int c) {
    float v = a.conv_b ? a.conv_b[c] : 0.f;
    for (int j = 0; j < a.taps; ++j) {
      float x = 0.f;
      if (j <= i) x = __bfloat162float(a.proj[(m - j) * a.ldp + c]);
      else if (p0 + i - j >= 0) x = tail[(int64_t)((p0 + i - j) % a.taps) * a.C + c];
      v += a.conv_w[(int64_t)c * a.taps + a.taps - 1 - j] * x;
    }
    return silu(v);
  };
  for (int u = warp; u < 2 * a.KH; u += nw) {
    const bool isk = u >= a.KH;
    const int h = isk ? u - a.KH : u;
    const int c0 = (isk ? a.k_off : a.q_off) + h * a.dk;
    __nv_bfloat16* out = (isk ? a.k : a.q) + m * (int64_t)a.KH * a.DKp + (int64_t)h * a.DKp;
    float ss = 0.f;
    for (int e = lane; e < a.DKp; e += 32) {
      const __nv_bfloat16 b = __float2bfloat16_rn(e < a.dk ? conv(c0 + e) : 0.f);
      out[e] = b;
      const float f = __bfloat162float(b);
      ss += f * f;
    }
#pragma unroll
    for (int o = 16; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (lane == 0)
      (isk ? a.rk : a.rq)[m * a.KH + h] = a.delta ? (isk ? 1.f : rsqrtf((float)a.dk)) / sqrtf(ss + 1e-6f) : 1.f;
  }
  for (int x = threadIdx.x; x < a.H * a.dvp; x += blockDim.x) {
    const int h = x / a.dvp, e = x - h * a.dvp;
    a.v[m * (int64_t)a.H * a.dvp + x] = __float2bfloat16_rn(e < a.dv ? conv(a.v_off + h * a.dv + e) : 0.f);
  }
}

// pairs of f32 in one 64-bit register: Blackwell's packed f32 arithmetic, rounded like the scalar one
__device__ __forceinline__ uint64_t pack2(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t widen2(uint32_t v) { return pack2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u)); }
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Sizes in multiples of 8: a thread takes 4 neighbouring channels of 32 tokens and slides over
// them.  Same outputs.
constexpr int CONV_TOK = 32;
constexpr int CV = 4;  // neighbouring channels of a thread
template <int TAPS>
__global__ void __launch_bounds__(128, 6) k_conv_chunk(ChunkArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int chunk = blockIdx.y / (CT / CONV_TOK), sub = blockIdx.y % (CT / CONV_TOK);
  const int t_lo = sub * CONV_TOK, t_hi = min(t_lo + CONV_TOK, a.chunk_len[chunk]);
  if (t_lo >= t_hi) return;
  const int64_t m0 = a.chunk_tok[chunk] + t_lo;
  const int row = a.rows.tok_row[m0];
  const int64_t p0 = row_pos0(a.rows, row);
  const int i0 = (int)(m0 - a.rows.start[row]);
  const int c = (blockIdx.x * 128 + threadIdx.x) * CV;
  const bool live = c < a.C;
  const int cc = live ? c : 0;
  const float* tail = a.tail + (int64_t)a.rows.slot[row] * a.taps * a.C + cc;
  uint64_t w[TAPS][CV / 2], bias[CV / 2];  // channel pairs
#pragma unroll
  for (int e = 0; e < CV / 2; ++e) {
    bias[e] = a.conv_b ? pack2(a.conv_b[cc + 2 * e], a.conv_b[cc + 2 * e + 1]) : 0;
    const float* t0 = a.conv_w + (int64_t)(cc + 2 * e) * TAPS;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j][e] = pack2(t0[TAPS - 1 - j], t0[2 * TAPS - 1 - j]);
  }
  // x[TAPS - 1 + i]: the input of the group's token i; x[TAPS - 1 - j]: the one j tokens before the group
  constexpr int G = 4;
  uint64_t x[TAPS - 1 + G][CV / 2];
  static_assert(CV == 4, "two channel pairs");
#pragma unroll
  for (int j = 1; j < TAPS; ++j) {
    uint64_t* v = x[TAPS - 1 - j];
    v[0] = v[1] = 0;
    if (j <= i0) {
      const uint2 r = *(const uint2*)(a.proj + (m0 - j) * a.ldp + cc);
      v[0] = widen2(r.x); v[1] = widen2(r.y);
    } else if (p0 + i0 - j >= 0) {
      const float* tp = tail + (int64_t)((p0 + i0 - j) % a.taps) * a.C;
      v[0] = pack2(tp[0], tp[1]); v[1] = pack2(tp[2], tp[3]);
    }
  }
  // where these channels go
  const int qk = a.KH * a.dk;
  __nv_bfloat16* out;
  float* rn = nullptr;
  int64_t ld;
  float f = 1.f;
  if (c >= a.v_off && c < a.v_off + a.H * a.dv) {
    const int h = (c - a.v_off) / a.dv, e = (c - a.v_off) - h * a.dv;
    out = a.v + (int64_t)h * a.dvp + e; ld = (int64_t)a.H * a.dvp;
  } else {
    const bool isk = c >= a.k_off && c < a.k_off + qk;
    const int off = c - (isk ? a.k_off : a.q_off);
    const int h = off / a.dk, e = off - h * a.dk;
    out = (isk ? a.k : a.q) + (int64_t)h * a.DKp + e; ld = (int64_t)a.KH * a.DKp;
    if (e == 0) rn = (isk ? a.rk : a.rq) + h;
    if (!isk) f = rsqrtf((float)a.dk);
  }
  const int lanes = a.dk / CV;  // threads of a head: a power of two dividing the warp
  const bool normed = __any_sync(0xffffffffu, a.delta && c < a.v_off);  // this warp has query or key channels
  const __nv_bfloat16* pin = a.proj + m0 * a.ldp + cc;
  __nv_bfloat16* po = out + m0 * ld;
  float* pn = rn ? rn + m0 * a.KH : nullptr;
  const uint64_t nlog2e = pack2(-1.4426950408889634f, -1.4426950408889634f), one2 = pack2(1.f, 1.f);
  const int n = live ? t_hi - t_lo : 0;  // tokens this thread stores
  int t = 0;
  uint2 raw[G];
  auto fetch = [&]() {
#pragma unroll
    for (int i = 0; i < G; ++i) {
      raw[i] = t + i < t_hi - t_lo ? *(const uint2*)pin : make_uint2(0, 0);
      pin += a.ldp;
    }
  };
  fetch();
  for (; t < t_hi - t_lo;) {
#pragma unroll
    for (int i = 0; i < G; ++i) { x[TAPS - 1 + i][0] = widen2(raw[i].x); x[TAPS - 1 + i][1] = widen2(raw[i].y); }
    t += G;
    fetch();  // the next group's inputs are on the way while this one is computed
#pragma unroll
    for (int i = 0; i < G; ++i) {
      uint32_t o[2];
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint64_t v = bias[e];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) v = fma2(w[j][e], x[TAPS - 1 + i - j][e], v);
        // silu: v / (1 + 2^(-v log2 e)), rounded to bf16 at once
        const float2 z = unpack2(mul2(v, nlog2e));
        const float2 d = unpack2(add2(pack2(ex2(z.x), ex2(z.y)), one2));
        const float2 y = unpack2(mul2(v, pack2(rcp(d.x), rcp(d.y))));
        const __nv_bfloat162 h2 = __floats2bfloat162_rn(y.x, y.y);
        o[e] = *(const uint32_t*)&h2;
      }
      if (normed) {
        const uint64_t a0 = widen2(o[0]), a1 = widen2(o[1]);
        const float2 q = unpack2(fma2(a1, a1, mul2(a0, a0)));
        ss = q.x + q.y;
      }
      const bool in = t - G + i < n;
      if (in) *(uint2*)po = make_uint2(o[0], o[1]);
      po += ld;
      if (normed) {
#pragma unroll
        for (int s = 16; s; s >>= 1)
          if (s < lanes) ss += __shfl_xor_sync(0xffffffffu, ss, s);
      }
      if (pn) {
        if (in) *pn = normed ? f * rsqrtf(ss + 1e-6f) : 1.f;
        pn += a.KH;
      }
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
      for (int e = 0; e < CV / 2; ++e) x[j][e] = x[j + G][e];
  }
}

// log decays and write strengths
__global__ void k_gates(ChunkArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int64_t n = a.rows.M * a.H;
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t m = i / a.H;
    const int h = (int)(i - m * a.H);
    const float* sp = a.small + m * a.ld_small;
    if (a.key_decay) {
      a.co[i] = 1.f / (1.f + expf(-sp[h]));
      continue;
    }
    const float dt = softplus(sp[a.delta ? a.H + h : h] + a.dt_bias[h]);
    a.gl[i] = -expf(a.a_log[h]) * dt;
    a.co[i] = a.delta ? 1.f / (1.f + expf(-sp[h])) : dt;
  }
}

// the last inputs of the convolution, at their position modulo taps
__global__ void k_conv_tail_ring(ChunkArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int row = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= a.C) return;
  const int64_t s0 = a.rows.start[row], p0 = row_pos0(a.rows, row);
  const int len = (int)(a.rows.start[row + 1] - s0);
  float* tail = a.tail + (int64_t)a.rows.slot[row] * a.taps * a.C;
  for (int i = max(0, len - a.taps + 1); i < len; ++i)
    tail[(int64_t)((p0 + i) % a.taps) * a.C + c] = __bfloat162float(a.proj[(s0 + i) * a.ldp + c]);
}

// ------------------------------------------------------------------ gates of a chunk ----
struct alignas(16) Gates {  // (pairs are read as 8-byte words)
  float G[CT];           // running sum of the log decays, base 2
  float co[CT], rk[CT];  // beta or dt; unit-norm factor of the key
  float rq[CT];          // unit-norm factor of the query
  float ek[CT], eq[CT];  // e^{G_t} times those factors
  float f[CT];           // what scales token t's write in the state after the chunk: e^{G_last - G_t} rk (ssd: and dt)
  float whole;           // e^{G_last}
};
// by one warp: lane l takes tokens 2 l and 2 l + 1
__device__ __forceinline__ void load_gates(const ChunkArgs& a, int chunk, int h, int kh, Gates* g, int lane) {
  const int len = a.chunk_len[chunk];
  const int64_t m0 = a.chunk_tok[chunk];
  float l[2], co[2], rq[2], rk[2];
#pragma unroll
  for (int b = 0; b < 2; ++b) {
    const int t = 2 * lane + b;
    const bool in = t < len;
    if (a.log_decay) {
      l[b] = in ? a.log_decay[h] * 1.4426950408889634f : 0.f;
      co[b] = rq[b] = rk[b] = in ? 1.f : 0.f;
      continue;
    }
    l[b] = in ? a.gl[(m0 + t) * a.H + h] * 1.4426950408889634f : 0.f;
    co[b] = in ? a.co[(m0 + t) * a.H + h] : 0.f;
    rq[b] = in ? a.rq[(m0 + t) * a.KH + kh] : 0.f;
    rk[b] = in ? a.rk[(m0 + t) * a.KH + kh] : 0.f;
  }
  const float sum = l[0] + l[1];
  float inc = sum;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float v = __shfl_up_sync(0xffffffffu, inc, o);
    if (lane >= o) inc += v;
  }
  const float last = __shfl_sync(0xffffffffu, inc, 31);
#pragma unroll
  for (int b = 0; b < 2; ++b) {
    const int t = 2 * lane + b;
    const float G = b ? inc : inc - l[1];
    g->G[t] = G;
    g->co[t] = co[b];
    g->rq[t] = rq[b];
    g->rk[t] = rk[b];
    g->eq[t] = pow2(G) * rq[b];
    g->ek[t] = pow2(G) * rk[b];
    g->f[t] = pow2(last - G) * rk[b] * (a.delta ? 1.f : co[b]);
  }
  if (lane == 0) g->whole = pow2(last);
}

// ------------------------------------------------------------------ T = (I + A)^-1 ----
template <int DK>
__global__ void __launch_bounds__(128) k_delta_solve(ChunkArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  constexpr int LK = DK + 8, LA = CHUNK_LD;
  extern __shared__ __align__(16) uint8_t smem[];
  float* A = (float*)smem;                       // [64][LA]
  float* X = A + CT * LA;                        // [64][LA]
  __nv_bfloat16* K = (__nv_bfloat16*)X;          // [64][LK], dead before X is written
  __shared__ Gates g;
  const int chunk = blockIdx.x, h = blockIdx.y, kh = h / (a.H / a.KH);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int len = a.chunk_len[chunk];
  const int64_t m0 = a.chunk_tok[chunk];
  const uint32_t ku = sm_u32(K);
  const int ch = a.DKp / 8;
  for (int i = tid; i < CT * (DK / 8); i += 128) {
    const int r = i / (DK / 8), c = i - r * (DK / 8);
    const bool in = r < len && c < ch;
    cp_async16(ku + (uint32_t)(r * LK + c * 8) * 2u, a.k + (m0 + (in ? r : 0)) * (int64_t)a.KH * a.DKp + (int64_t)kh * a.DKp + (in ? c * 8 : 0),
               in ? 16 : 0);
  }
  if (warp == 0) load_gates(a, chunk, h, kh, &g, lane);
  cp_async_wait_all();
  __syncthreads();
  float acc[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < DK; kk += 16) {
    uint32_t fa[4], fb[4];
    frag_a(ku, LK, warp * 16, kk, lane, fa);
#pragma unroll
    for (int j = 0; j < 8; j += 2) {
      frag_b_nk(ku, LK, kk, j * 8, lane, fb);
      mma_bf16(acc[j], fa[0], fa[1], fa[2], fa[3], fb[0], fb[1]);
      mma_bf16(acc[j + 1], fa[0], fa[1], fa[2], fa[3], fb[2], fb[3]);
    }
  }
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = warp * 16 + (lane >> 2) + 8 * (e >> 1), s = j * 8 + (lane & 3) * 2 + (e & 1);
      A[t * LA + s] = s < t ? g.co[t] * g.rk[t] * g.rk[s] * pow2(g.G[t] - g.G[s]) * acc[j][e] : 0.f;
    }
  __syncthreads();
  invert_unit_lower(A, X, tid, 128);
  __nv_bfloat16* out = a.T + ((int64_t)chunk * a.H + h) * 2 * CT * CT;
  for (int i = tid; i < CT * CT / 2; i += 128) {
    const int r = i / (CT / 2), c = (i - r * (CT / 2)) * 2;
    uint32_t hi, lo;
    split2(X[r * LA + c], X[r * LA + c + 1], hi, lo);
    *(uint32_t*)(out + r * CT + c) = hi;
    *(uint32_t*)(out + CT * CT + r * CT + c) = lo;
  }
}

// ------------------------------------------------------------------ the walk ----------
// Regions are reused inside a chunk so that two blocks share an SM: P takes Q's place, R and then U
// take V's (and one more for the remainders), U' takes T's.
template <int DK>
struct DeltaSmem {
  static constexpr int LK = DK + 8;
  static constexpr uint32_t EBYTES = CT * LE * 2;
  static constexpr uint32_t Q = 0, P = 0;                        // [64][LK] | [2][64][LT]
  static constexpr uint32_t K = (CT * LK > 2 * CT * LT ? CT * LK : 2 * CT * LT) * 2;
  static constexpr uint32_t V = K + CT * LK * 2;                 // [64][LE]
  static constexpr uint32_t RL = V + EBYTES;                     // [64][LE]
  static constexpr uint32_t T = RL + EBYTES;                     // [2][64][LT] | U' [2][64][LE]
  static constexpr uint32_t UP = T;
  static constexpr uint32_t S = T + 2 * EBYTES;                  // [2][DK][LE]
  static constexpr uint32_t GATES = S + 2 * DK * LE * 2;
  static constexpr uint32_t BYTES = GATES + 2 * sizeof(Gates);
  static_assert(LE == LT, "T and U' share a region");
};

template <int DK>
__global__ void __launch_bounds__(256, 2) k_delta_scan(ChunkArgs a) {
  using L = DeltaSmem<DK>;
  constexpr int LK = L::LK;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  extern __shared__ __align__(16) uint8_t smem[];
  const uint32_t base = sm_u32(smem);
  Gates* gates = (Gates*)(smem + L::GATES);
  const int e0 = blockIdx.x * EB, h = blockIdx.y, row = blockIdx.z, kh = h / (a.H / a.KH);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int wm = warp & 3, wn = warp >> 2;            // this warp's 16 tokens and 32 columns
  const int r_in = lane >> 2, cq = (lane & 3) * 2;
  const int c0 = a.row_chunk[row], c1 = a.row_chunk[row + 1];
  const bool first = row_pos0(a.rows, row) == 0;
  const int vw = min(EB, a.dvp - e0);                 // columns that exist (multiple of 8)

  auto load = [&](int chunk) {
    const int len = a.chunk_len[chunk];
    const int64_t m0 = a.chunk_tok[chunk];
    const uint32_t b = base;
    const int ch = a.DKp / 8;
    for (int i = tid; i < CT * (DK / 8); i += 256) {
      const int r = i / (DK / 8), c = i - r * (DK / 8);
      const bool in = r < len && c < ch;
      const int64_t o = (m0 + (in ? r : 0)) * a.ldq + (int64_t)kh * a.DKp + (in ? c * 8 : 0);
      const uint32_t d = (uint32_t)(r * LK + c * 8) * 2u;
      cp_async16(b + L::Q + d, a.q + o, in ? 16 : 0);
      cp_async16(b + L::K + d, a.k + o, in ? 16 : 0);
    }
    for (int i = tid; i < CT * (EB / 8); i += 256) {
      const int r = i / (EB / 8), c = i - r * (EB / 8);
      const bool in = r < len && c * 8 < vw;
      cp_async16(b + L::V + (uint32_t)(r * LE + c * 8) * 2u,
                 a.v + (m0 + (in ? r : 0)) * a.ldv + (int64_t)h * a.dvp + (in ? e0 + c * 8 : 0), in ? 16 : 0);
    }
    {
      const __nv_bfloat16* t = a.T + ((int64_t)chunk * a.H + h) * 2 * CT * CT;
      for (int i = tid; i < 2 * CT * (CT / 8); i += 256) {
        const int r = i / (CT / 8), c = i - r * (CT / 8);
        cp_async16(b + L::T + (uint32_t)(r * LT + c * 8) * 2u, t + r * CT + c * 8, 16);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(c0);
  if (warp == 7) load_gates(a, c0, h, kh, &gates[0], lane);

  // the state: DK / 16 row tiles over the warps
  constexpr int SN = DK == 128 ? 8 : 4;               // 8-column tiles a warp holds
  const int sr = DK == 128 ? warp * 16 : wm * 16, sc = DK == 128 ? 0 : wn * 32;
  float S[SN][4];
  float* Sg = a.S + ((int64_t)a.rows.slot[row] * a.H + h) * a.dk * a.dvs;
#pragma unroll
  for (int j = 0; j < SN; ++j)
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int r = sr + r_in + 8 * b, c = e0 + sc + j * 8 + cq;
      float2 v = make_float2(0.f, 0.f);
      if (!first && r < a.dk && c < a.dvs) v = *(const float2*)(Sg + (int64_t)r * a.dvs + c);
      S[j][2 * b] = v.x; S[j][2 * b + 1] = v.y;
    }
  auto publish_state = [&]() {
#pragma unroll
    for (int j = 0; j < SN; ++j)
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        uint32_t hi, lo;
        split2(S[j][2 * b], S[j][2 * b + 1], hi, lo);
        const uint32_t o = (uint32_t)((sr + r_in + 8 * b) * LE + sc + j * 8 + cq) * 2u;
        *(uint32_t*)(smem + L::S + o) = hi;
        *(uint32_t*)(smem + L::S + DK * LE * 2 + o) = lo;
      }
  };
  publish_state();

  for (int c = c0; c < c1; ++c) {
    const int stage = (c - c0) & 1;
    const uint32_t b = base;
    const Gates& g = gates[stage];
    cp_async_wait_all();
    __syncthreads();  // tiles, gates and state of this chunk are in place
    if (c + 1 < c1 && warp == 7) load_gates(a, c + 1, h, kh, &gates[stage ^ 1], lane);
    const int t0 = wm * 16 + r_in;                    // this thread's tokens: t0 and t0 + 8
    float qs[4][4];                                    // Q S0
    {
      float ks[4][4], qk[4][4];                        // K S0 (delta), Q K^T
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) qs[j][e] = ks[j][e] = qk[j][e] = 0.f;
      const bool below = wn * 32 <= wm * 16 + 15;      // some key of this tile is visible to some token
#pragma unroll
      for (int kk = 0; kk < DK; kk += 16) {
        uint32_t fq[4], fk[4], fb[4];
        frag_a(b + L::Q, LK, wm * 16, kk, lane, fq);
        frag_a(b + L::K, LK, wm * 16, kk, lane, fk);
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
#pragma unroll
          for (int part = 0; part < 2; ++part) {
            frag_b_kn(base + L::S + (uint32_t)(part * DK * LE * 2), LE, kk, wn * 32 + j * 8, lane, fb);
            mma_bf16(qs[j], fq[0], fq[1], fq[2], fq[3], fb[0], fb[1]);
            mma_bf16(qs[j + 1], fq[0], fq[1], fq[2], fq[3], fb[2], fb[3]);
            mma_bf16(ks[j], fk[0], fk[1], fk[2], fk[3], fb[0], fb[1]);
            mma_bf16(ks[j + 1], fk[0], fk[1], fk[2], fk[3], fb[2], fb[3]);
          }
          if (below) {
            frag_b_nk(b + L::K, LK, kk, wn * 32 + j * 8, lane, fb);
            mma_bf16(qk[j], fq[0], fq[1], fq[2], fq[3], fb[0], fb[1]);
            mma_bf16(qk[j + 1], fq[0], fq[1], fq[2], fq[3], fb[2], fb[3]);
          }
        }
      }
      __syncthreads();  // Q and the old state are read
      // P and R (or the state's addends) into shared memory, split
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int t = t0 + 8 * x, n = wn * 32 + j * 8 + cq;
          float p[2];
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            const int s = n + y;
            p[y] = s <= t ? pow2(g.G[t] - g.G[s]) * g.rq[t] * g.rk[s] * qk[j][2 * x + y] : 0.f;
          }
          uint32_t hi, lo;
          split2(p[0], p[1], hi, lo);
          const uint32_t o = (uint32_t)(t * LT + n) * 2u;
          *(uint32_t*)(smem + L::P + o) = hi;
          *(uint32_t*)(smem + L::P + CT * LT * 2 + o) = lo;
          const float2 v = __bfloat1622float2(*(const __nv_bfloat162*)(smem + L::V + (uint32_t)(t * LE + n) * 2u));
          const uint32_t oe = (uint32_t)(t * LE + n) * 2u;
          const float f = g.ek[t];
          split2(g.co[t] * (v.x - f * ks[j][2 * x]), g.co[t] * (v.y - f * ks[j][2 * x + 1]), hi, lo);
          *(uint32_t*)(smem + L::V + oe) = hi;  // (this thread's own value of V)
          *(uint32_t*)(smem + L::RL + oe) = lo;
        }
    }
    __syncthreads();
    {
      // U = T R
      float u[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) u[j][0] = u[j][1] = u[j][2] = u[j][3] = 0.f;
      for (int kk = 0; kk <= wm * 16; kk += 16) {
        uint32_t th[4], tl[4], fh[4], fl[4];
        frag_a(b + L::T, LT, wm * 16, kk, lane, th);
        frag_a(b + L::T + CT * LT * 2, LT, wm * 16, kk, lane, tl);
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          frag_b_kn(base + L::V, LE, kk, wn * 32 + j * 8, lane, fh);
          frag_b_kn(base + L::RL, LE, kk, wn * 32 + j * 8, lane, fl);
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            mma_bf16(u[j + y], th[0], th[1], th[2], th[3], fh[2 * y], fh[2 * y + 1]);
            mma_bf16(u[j + y], th[0], th[1], th[2], th[3], fl[2 * y], fl[2 * y + 1]);
            mma_bf16(u[j + y], tl[0], tl[1], tl[2], tl[3], fh[2 * y], fh[2 * y + 1]);
          }
        }
      }
      __syncthreads();  // T and R are read: U' and U take their places
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int t = t0 + 8 * x;
          const uint32_t oe = (uint32_t)(t * LE + wn * 32 + j * 8 + cq) * 2u;
          uint32_t hi, lo;
          split2(u[j][2 * x], u[j][2 * x + 1], hi, lo);
          *(uint32_t*)(smem + L::V + oe) = hi;
          *(uint32_t*)(smem + L::RL + oe) = lo;
          const float f = g.f[t];
          split2(f * u[j][2 * x], f * u[j][2 * x + 1], hi, lo);
          *(uint32_t*)(smem + L::UP + oe) = hi;
          *(uint32_t*)(smem + L::UP + CT * LE * 2 + oe) = lo;
        }
      __syncthreads();
    }
    // O = e^G rq (Q S0) + P U
    {
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const float f = g.eq[t0 + 8 * x];
#pragma unroll
        for (int j = 0; j < 4; ++j) { qs[j][2 * x] *= f; qs[j][2 * x + 1] *= f; }
      }
      for (int kk = 0; kk <= wm * 16; kk += 16) {
        uint32_t ph[4], pl[4], fh[4], fl[4];
        frag_a(base + L::P, LT, wm * 16, kk, lane, ph);
        frag_a(base + L::P + CT * LT * 2, LT, wm * 16, kk, lane, pl);
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          frag_b_kn(base + L::V, LE, kk, wn * 32 + j * 8, lane, fh);
          frag_b_kn(base + L::RL, LE, kk, wn * 32 + j * 8, lane, fl);
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            mma_bf16(qs[j + y], ph[0], ph[1], ph[2], ph[3], fh[2 * y], fh[2 * y + 1]);
            mma_bf16(qs[j + y], pl[0], pl[1], pl[2], pl[3], fh[2 * y], fh[2 * y + 1]);
            mma_bf16(qs[j + y], ph[0], ph[1], ph[2], ph[3], fl[2 * y], fl[2 * y + 1]);
          }
        }
      }
      const int len = a.chunk_len[c];
      const int64_t m0 = a.chunk_tok[c];
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int t = t0 + 8 * x;
        if (t >= len) continue;
        float* o = a.o + (m0 + t) * (int64_t)a.H * a.dvs + (int64_t)h * a.dvs + e0;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int n = wn * 32 + j * 8 + cq;
          if (e0 + n >= a.dvs) continue;
          const float2 r = make_float2(qs[j][2 * x], qs[j][2 * x + 1]);
          *(float2*)(o + n) = r;
        }
      }
    }
    // S = e^{G_last} S + K^T U'
    {
      const float f = g.whole;
#pragma unroll
      for (int j = 0; j < SN; ++j) { S[j][0] *= f; S[j][1] *= f; S[j][2] *= f; S[j][3] *= f; }
#pragma unroll
      for (int kk = 0; kk < CT; kk += 16) {
        uint32_t fk[4], fb[4];
        frag_a_t(b + L::K, LK, sr, kk, lane, fk);
#pragma unroll
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int j = 0; j < SN; j += 2) {
            frag_b_kn(base + L::UP + (uint32_t)(part * CT * LE * 2), LE, kk, sc + j * 8, lane, fb);
            mma_bf16(S[j], fk[0], fk[1], fk[2], fk[3], fb[0], fb[1]);
            mma_bf16(S[j + 1], fk[0], fk[1], fk[2], fk[3], fb[2], fb[3]);
          }
      }
    }
    if (c + 1 < c1) {
      __syncthreads();  // the chunk's tiles are read
      load(c + 1);
      publish_state();
    }
  }
#pragma unroll
  for (int j = 0; j < SN; ++j)
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int r = sr + r_in + 8 * b, c = e0 + sc + j * 8 + cq;
      if (r < a.dk && c < a.dvs) *(float2*)(Sg + (int64_t)r * a.dvs + c) = make_float2(S[j][2 * b], S[j][2 * b + 1]);
    }
}

// The state space needs no solve, and its values are exact as bf16: P stays in registers from the
// score product to the value product, and the writes' scales go onto the key operand.
template <int DK>
struct SsdSmem {
  static constexpr int LK = DK + 8;
  static constexpr uint32_t Q = 0, K = CT * LK * 2, V = K + CT * LK * 2;
  static constexpr uint32_t S = V + CT * LE * 2;                 // [2][DK][LE]
  static constexpr uint32_t GATES = S + 2 * DK * LE * 2;
  static constexpr uint32_t BYTES = GATES + 2 * sizeof(Gates);
};

template <int DK>
__global__ void __launch_bounds__(256, 2) k_ssd_scan(ChunkArgs a) {
  using L = SsdSmem<DK>;
  constexpr int LK = L::LK;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  extern __shared__ __align__(16) uint8_t smem[];
  const uint32_t base = sm_u32(smem);
  Gates* gates = (Gates*)(smem + L::GATES);
  const int e0 = blockIdx.x * EB, h = blockIdx.y, row = blockIdx.z, kh = h / (a.H / a.KH);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int wm = warp & 3, wn = warp >> 2;            // this warp's 16 tokens and 32 columns
  const int r_in = lane >> 2, cq = (lane & 3) * 2;
  const int c0 = a.row_chunk[row], c1 = a.row_chunk[row + 1];
  const bool first = row_pos0(a.rows, row) == 0;
  const int vw = min(EB, a.dvp - e0);

  auto load = [&](int chunk) {
    const int len = a.chunk_len[chunk];
    const int64_t m0 = a.chunk_tok[chunk];
    const int ch = a.DKp / 8;
    for (int i = tid; i < CT * (DK / 8); i += 256) {
      const int r = i / (DK / 8), c = i - r * (DK / 8);
      const bool in = r < len && c < ch;
      const int64_t o = (m0 + (in ? r : 0)) * a.ldq + (int64_t)kh * a.DKp + (in ? c * 8 : 0);
      const uint32_t d = (uint32_t)(r * LK + c * 8) * 2u;
      cp_async16(base + L::Q + d, a.q + o, in ? 16 : 0);
      cp_async16(base + L::K + d, a.k + o, in ? 16 : 0);
    }
    for (int i = tid; i < CT * (EB / 8); i += 256) {
      const int r = i / (EB / 8), c = i - r * (EB / 8);
      const bool in = r < len && c * 8 < vw;
      cp_async16(base + L::V + (uint32_t)(r * LE + c * 8) * 2u,
                 a.v + (m0 + (in ? r : 0)) * a.ldv + (int64_t)h * a.dvp + (in ? e0 + c * 8 : 0), in ? 16 : 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(c0);
  if (warp == 7) load_gates(a, c0, h, kh, &gates[0], lane);

  constexpr int SN = DK == 128 ? 8 : 4;
  const int sr = DK == 128 ? warp * 16 : wm * 16, sc = DK == 128 ? 0 : wn * 32;
  float S[SN][4];
  float* Sg = a.S + ((int64_t)a.rows.slot[row] * a.H + h) * a.dk * a.dvs;
#pragma unroll
  for (int j = 0; j < SN; ++j)
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int r = sr + r_in + 8 * b, c = e0 + sc + j * 8 + cq;
      float2 v = make_float2(0.f, 0.f);
      if (!first && r < a.dk && c < a.dvs) v = *(const float2*)(Sg + (int64_t)r * a.dvs + c);
      S[j][2 * b] = v.x; S[j][2 * b + 1] = v.y;
    }
  auto publish_state = [&]() {
#pragma unroll
    for (int j = 0; j < SN; ++j)
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        uint32_t hi, lo;
        split2(S[j][2 * b], S[j][2 * b + 1], hi, lo);
        const uint32_t o = (uint32_t)((sr + r_in + 8 * b) * LE + sc + j * 8 + cq) * 2u;
        *(uint32_t*)(smem + L::S + o) = hi;
        *(uint32_t*)(smem + L::S + DK * LE * 2 + o) = lo;
      }
  };
  publish_state();
  const float dsk = a.dskip ? a.dskip[h] : 0.f;
  const int t0 = wm * 16 + r_in;                      // this thread's tokens: t0 and t0 + 8

  for (int c = c0; c < c1; ++c) {
    const Gates& g = gates[(c - c0) & 1];
    cp_async_wait_all();
    __syncthreads();  // tiles, gates and state of this chunk are in place
    if (c + 1 < c1 && warp == 7) load_gates(a, c + 1, h, kh, &gates[(c + 1 - c0) & 1], lane);
    float o[4][4], qk[8][4];                           // C S0, then the output; C B^T of keys 0 .. wm * 16 + 15
#pragma unroll
    for (int j = 0; j < 4; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) qk[j][0] = qk[j][1] = qk[j][2] = qk[j][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < DK; kk += 16) {
      uint32_t fq[4], fb[4];
      frag_a(base + L::Q, LK, wm * 16, kk, lane, fq);
#pragma unroll
      for (int j = 0; j < 4; j += 2)
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          frag_b_kn(base + L::S + (uint32_t)(part * DK * LE * 2), LE, kk, wn * 32 + j * 8, lane, fb);
          mma_bf16(o[j], fq[0], fq[1], fq[2], fq[3], fb[0], fb[1]);
          mma_bf16(o[j + 1], fq[0], fq[1], fq[2], fq[3], fb[2], fb[3]);
        }
#pragma unroll
      for (int j = 0; j < 8; j += 2)
        if (j <= 2 * wm) {
          frag_b_nk(base + L::K, LK, kk, j * 8, lane, fb);
          mma_bf16(qk[j], fq[0], fq[1], fq[2], fq[3], fb[0], fb[1]);
          mma_bf16(qk[j + 1], fq[0], fq[1], fq[2], fq[3], fb[2], fb[3]);
        }
    }
    const float G0 = g.G[t0], G1 = g.G[t0 + 8];
    {
      const float f0 = g.eq[t0], f1 = g.eq[t0 + 8];
#pragma unroll
      for (int j = 0; j < 4; ++j) { o[j][0] *= f0; o[j][1] *= f0; o[j][2] *= f1; o[j][3] *= f1; }
    }
    // o += P x: the scores' accumulator layout is the operand layout of the next product
#pragma unroll
    for (int kt = 0; kt < 4; ++kt)
      if (kt <= wm) {
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int j = 2 * kt + half, s = j * 8 + cq;
          const float2 Gs = *(const float2*)(g.G + s), cs = *(const float2*)(g.co + s);
          float p[4] = {qk[j][0] * pow2(G0 - Gs.x) * cs.x, qk[j][1] * pow2(G0 - Gs.y) * cs.y, qk[j][2] * pow2(G1 - Gs.x) * cs.x,
                        qk[j][3] * pow2(G1 - Gs.y) * cs.y};
          if (kt == wm) {
            p[0] = s <= t0 ? p[0] : 0.f;
            p[1] = s + 1 <= t0 ? p[1] : 0.f;
            p[2] = s <= t0 + 8 ? p[2] : 0.f;
            p[3] = s + 1 <= t0 + 8 ? p[3] : 0.f;
          }
          split2(p[0], p[1], ph[2 * half], pl[2 * half]);
          split2(p[2], p[3], ph[2 * half + 1], pl[2 * half + 1]);
        }
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          uint32_t fb[4];
          frag_b_kn(base + L::V, LE, kt * 16, wn * 32 + j * 8, lane, fb);
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            mma_bf16(o[j + y], ph[0], ph[1], ph[2], ph[3], fb[2 * y], fb[2 * y + 1]);
            mma_bf16(o[j + y], pl[0], pl[1], pl[2], pl[3], fb[2 * y], fb[2 * y + 1]);
          }
        }
      }
    {
      const int len = a.chunk_len[c];
      const int64_t m0 = a.chunk_tok[c];
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int t = t0 + 8 * x;
        if (t >= len) continue;
        float* og = a.o + (m0 + t) * (int64_t)a.H * a.dvs + (int64_t)h * a.dvs + e0;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int n = wn * 32 + j * 8 + cq;
          if (e0 + n >= a.dvs) continue;
          const float2 v = __bfloat1622float2(*(const __nv_bfloat162*)(smem + L::V + (uint32_t)(t * LE + n) * 2u));
          *(float2*)(og + n) = make_float2(o[j][2 * x] + dsk * v.x, o[j][2 * x + 1] + dsk * v.y);
        }
      }
    }
    // S = e^{G_last} S + (f B)^T x
    {
      const float f = g.whole;
#pragma unroll
      for (int j = 0; j < SN; ++j) { S[j][0] *= f; S[j][1] *= f; S[j][2] *= f; S[j][3] *= f; }
#pragma unroll
      for (int kk = 0; kk < CT; kk += 16) {
        uint32_t fk[4], kh4[4], kl4[4], fb[4];
        frag_a_t(base + L::K, LK, sr, kk, lane, fk);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 w = *(const float2*)(g.f + kk + cq + 8 * (i >> 1));
          const float2 k = __bfloat1622float2(*(const __nv_bfloat162*)&fk[i]);
          split2(k.x * w.x, k.y * w.y, kh4[i], kl4[i]);
        }
#pragma unroll
        for (int j = 0; j < SN; j += 2) {
          frag_b_kn(base + L::V, LE, kk, sc + j * 8, lane, fb);
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            mma_bf16(S[j + y], kh4[0], kh4[1], kh4[2], kh4[3], fb[2 * y], fb[2 * y + 1]);
            mma_bf16(S[j + y], kl4[0], kl4[1], kl4[2], kl4[3], fb[2 * y], fb[2 * y + 1]);
          }
        }
      }
    }
    if (c + 1 < c1) {
      __syncthreads();  // tiles and old state are read
      load(c + 1);
      publish_state();
    }
  }
#pragma unroll
  for (int j = 0; j < SN; ++j)
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int r = sr + r_in + 8 * b, c = e0 + sc + j * 8 + cq;
      if (r < a.dk && c < a.dvs) *(float2*)(Sg + (int64_t)r * a.dvs + c) = make_float2(S[j][2 * b], S[j][2 * b + 1]);
    }
}

template <int DK, bool DELTA>
int launch_scan(cg_ctx* c, const ChunkArgs& a) {
  constexpr size_t smem = DELTA ? (size_t)DeltaSmem<DK>::BYTES : (size_t)SsdSmem<DK>::BYTES;
  static_assert(smem <= 113 * 1024, "two blocks per SM");
  auto kernel = DELTA ? k_delta_scan<DK> : k_ssd_scan<DK>;
  static PerDeviceFlag configured_on;
  bool& configured = configured_on.at(c->core->device);
  if (!configured) {
    CG_CUDA(c, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = true;
  }
  dim3 grid((unsigned)((a.dv + EB - 1) / EB), (unsigned)a.H, (unsigned)a.rows.rows);
  CG_CUDA(c, launch_kernel(c, kernel, grid, dim3(256), smem, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}
template <int DK>
int launch_solve(cg_ctx* c, const ChunkArgs& a) {
  constexpr size_t smem = (size_t)CT * 68 * 4 + std::max((size_t)CT * 68 * 4, (size_t)CT * (DK + 8) * 2);
  CG_CUDA(c, launch_kernel(c, k_delta_solve<DK>, dim3((unsigned)a.n_chunks, (unsigned)a.H), dim3(128), smem, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace

bool chunk_supported(int dk) { return dk <= 128; }

int k_launch_chunk_recurrence(cg_ctx* c, const ChunkArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  if (a.key_decay && !a.delta) return k_launch_channel_chunks(c, a);
  if (a.log_decay) return a.dk <= 64 ? launch_scan<64, false>(c, a) : launch_scan<128, false>(c, a);
  const int lanes = a.dk / CV;
  const bool fast = a.dk % 8 == 0 && a.dv % 8 == 0 && a.DKp == a.dk && (!a.delta || (lanes & (lanes - 1)) == 0) && a.taps >= 1 && a.taps <= 4;
  if (fast) {
    dim3 grid((unsigned)((a.C + 128 * CV - 1) / (128 * CV)), (unsigned)(a.n_chunks * (CT / CONV_TOK)));
    if (grid.y > 65535) return fail(c, CG_ERR_UNSUPPORTED, "recurrence: too many tokens in one portion");
    switch (a.taps) {
      case 1: CG_CUDA(c, launch_kernel(c, k_conv_chunk<1>, grid, dim3(128), 0, 1, a)); break;
      case 2: CG_CUDA(c, launch_kernel(c, k_conv_chunk<2>, grid, dim3(128), 0, 1, a)); break;
      case 3: CG_CUDA(c, launch_kernel(c, k_conv_chunk<3>, grid, dim3(128), 0, 1, a)); break;
      default: CG_CUDA(c, launch_kernel(c, k_conv_chunk<4>, grid, dim3(128), 0, 1, a)); break;
    }
  } else {
    CG_CUDA(c, launch_kernel(c, k_conv_chunk_any, dim3((unsigned)a.rows.M), dim3(256), 0, 1, a));
  }
  CG_LAUNCHED(c);
  CG_CUDA(c, launch_kernel(c, k_gates, dim3(grid_for(a.rows.M * a.H, 256)), dim3(256), 0, 1, a));
  CG_LAUNCHED(c);
  if (a.taps > 1) {
    CG_CUDA(c, launch_kernel(c, k_conv_tail_ring, dim3((unsigned)((a.C + 127) / 128), (unsigned)a.rows.rows), dim3(128), 0, 1, a));
    CG_LAUNCHED(c);
  }
  if (a.key_decay) return k_launch_channel_chunks(c, a);
  const bool small = a.dk <= 64;
  if (a.delta) {
    CG_TRY(small ? launch_solve<64>(c, a) : launch_solve<128>(c, a));
    return small ? launch_scan<64, true>(c, a) : launch_scan<128, true>(c, a);
  }
  return small ? launch_scan<64, false>(c, a) : launch_scan<128, false>(c, a);
}

}  // namespace cg
