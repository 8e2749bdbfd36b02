// lru.cu — Griffin's recurrent block: a diagonal linear recurrence whose decay and input gates are block
// diagonal maps of a short convolution's output, multiplied by a gelu branch.
//
//   u = conv(x + xb) + conv_b;  r = sigmoid(Ra u + ra_b), i = sigmoid(Ri u + ri_b), per block
//   ln a = -8 r softplus(lam);  S <- a S + sqrt(1 - a^2) i u;  out = S gelu(y + yb)
//
// Prompts: k_lru_conv, then the gates as one batch of block-diagonal products on the tensor cores whose
// epilogue leaves a and the gated input in f32, then a scan over time that composes eight tokens per
// thread and the segments of a tile through shared memory.  One token per row: everything in one kernel.
#include <algorithm>

#include "act.cuh"
#include "mixers.h"
#include "mma.cuh"

namespace cg {

namespace {

__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
// what u was when it entered the gates' products
__device__ __forceinline__ float as(float v, const float*) { return v; }
__device__ __forceinline__ float as(float v, const __nv_bfloat16*) { return __bfloat162float(__float2bfloat16_rn(v)); }
// a and sqrt(1 - a^2) i u from the gates before their sigmoids; f = -8 softplus(lam)
__device__ __forceinline__ float2 gate_pair(float zr, float zi, float f, float u) {
  const float la = f * sigmoid(zr);
  return make_float2(expf(la), sqrtf(-expm1f(2.f * la)) * sigmoid(zi) * u);
}

// The same for prompts in a bf16 context.  1 - a^2 = -(e^y - 1), y = 2 ln a, by its power series where
// 1 - e^y would lose digits.
__device__ __forceinline__ float2 gate_pair_fast(float zr, float zi, float f, float u) {
  const float la = f * sigmoid_fast(zr), y = 2.f * la, a = __expf(la);
  float p = fmaf(y, 1.f / 720.f, 1.f / 120.f);
  p = fmaf(p, y, 1.f / 24.f);
  p = fmaf(p, y, 1.f / 6.f);
  p = fmaf(p, y, 0.5f);
  p = fmaf(p, y, 1.f);
  const float q = y > -0.25f ? -y * p : 1.f - a * a;
  float s;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(s) : "f"(q));
  return make_float2(a, s * sigmoid_fast(zi) * u);
}

// the convolution at channel c of token i of its row, whose first position is p0
template <class TP>
__device__ __forceinline__ float conv_at(const LruArgs& a, const TP* x, int64_t m, int i, int64_t p0, int c, const float* tail) {
  float v = a.conv_b[c];
  const float b = a.xb[c];
  for (int j = 0; j < a.taps; ++j) {
    float t = 0.f;
    if (j <= i) t = ld(x + (m - j) * a.ldx + c) + b;
    else if (p0 + i - j >= 0) t = tail[(int64_t)((p0 + i - j) % a.taps) * a.W + c];
    v += a.conv_w[(int64_t)c * a.taps + a.taps - 1 - j] * t;
  }
  return v;
}

// One thread per channel and LC_TOK tokens.
constexpr int LC_TOK = 8;
template <class TP, class T>
__global__ void __launch_bounds__(128) k_lru_conv(LruArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int c = blockIdx.y * 128 + threadIdx.x;
  if (c >= a.W) return;
  const int64_t m0 = (int64_t)blockIdx.x * LC_TOK;
  const TP* x = (const TP*)a.x;
#pragma unroll
  for (int k = 0; k < LC_TOK; ++k) {
    const int64_t m = m0 + k;
    if (m >= a.rows.M) return;
    const int row = a.rows.tok_row[m];
    const float* tail = a.tail + (int64_t)a.rows.slot[row] * a.taps * a.W;
    st((T*)a.u + m * a.W + c, conv_at(a, x, m, (int)(m - a.rows.start[row]), row_pos0(a.rows, row), c, tail));
  }
}

// Channels in groups of 4 (bf16): a thread slides over 32 tokens of 4 channels, the next four tokens' inputs
// requested while four are summed.
constexpr int LV_TOK = 32;
__device__ __forceinline__ void widen4(uint2 r, float* v) {
  v[0] = __uint_as_float(r.x << 16); v[1] = __uint_as_float(r.x & 0xffff0000u);
  v[2] = __uint_as_float(r.y << 16); v[3] = __uint_as_float(r.y & 0xffff0000u);
}
template <int TAPS>
__global__ void __launch_bounds__(128) k_lru_conv_vec(LruArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  constexpr int G = 4, PER = RECUR_CHUNK / LV_TOK;
  const int chunk = blockIdx.x / PER, t_lo = (blockIdx.x % PER) * LV_TOK;
  const int n = min(LV_TOK, a.chunk_len[chunk] - t_lo), c = (blockIdx.y * 128 + threadIdx.x) * 4;
  if (n <= 0 || c >= a.W) return;
  const int64_t m0 = a.chunk_tok[chunk] + t_lo;
  const int row = a.rows.tok_row[m0], i0 = (int)(m0 - a.rows.start[row]);
  const int64_t p0 = row_pos0(a.rows, row);
  const float* tail = a.tail + (int64_t)a.rows.slot[row] * a.taps * a.W + c;
  const __nv_bfloat16* in = (const __nv_bfloat16*)a.x + m0 * a.ldx + c;
  float w[TAPS][4], xb[4], cb[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    xb[e] = a.xb[c + e];
    cb[e] = a.conv_b[c + e];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j][e] = a.conv_w[(int64_t)(c + e) * TAPS + TAPS - 1 - j];
  }
  // x[TAPS - 1 + i]: the input of the group's token i; x[TAPS - 1 - j]: the one j tokens before the group
  float x[TAPS - 1 + G][4];
#pragma unroll
  for (int j = 1; j < TAPS; ++j) {
    float* v = x[TAPS - 1 - j];
    v[0] = v[1] = v[2] = v[3] = 0.f;
    if (j <= i0) {
      widen4(*(const uint2*)(in - j * a.ldx), v);
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] += xb[e];
    } else if (p0 + i0 - j >= 0) {
      const float* tp = tail + (int64_t)((p0 + i0 - j) % TAPS) * a.W;
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = tp[e];
    }
  }
  uint2 raw[G];
  auto fetch = [&](int t) {
#pragma unroll
    for (int i = 0; i < G; ++i) raw[i] = t + i < n ? *(const uint2*)(in + (int64_t)(t + i) * a.ldx) : make_uint2(0, 0);
  };
  fetch(0);
  __nv_bfloat16* out = (__nv_bfloat16*)a.u + m0 * a.W + c;
  for (int t = 0; t < n; t += G) {
#pragma unroll
    for (int i = 0; i < G; ++i) {
      widen4(raw[i], x[TAPS - 1 + i]);
#pragma unroll
      for (int e = 0; e < 4; ++e) x[TAPS - 1 + i][e] += xb[e];
    }
    fetch(t + G);
#pragma unroll
    for (int i = 0; i < G; ++i) {
      float v[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[e] = cb[e];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) v[e] = fmaf(w[j][e], x[TAPS - 1 + i - j][e], v[e]);
      }
      const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
      if (t + i < n) *(uint2*)(out + (int64_t)(t + i) * a.W) = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) x[j][e] = x[j + G][e];
  }
}

// the last inputs of the convolution, at their position modulo taps
template <class TP>
__global__ void k_lru_tail(LruArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int row = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= a.W) return;
  const int64_t s0 = a.rows.start[row], p0 = row_pos0(a.rows, row);
  const int len = (int)(a.rows.start[row + 1] - s0);
  float* tail = a.tail + (int64_t)a.rows.slot[row] * a.taps * a.W;
  for (int i = max(0, len - a.taps + 1); i < len; ++i)
    tail[(int64_t)((p0 + i) % a.taps) * a.W + c] = ld((const TP*)a.x + (s0 + i) * a.ldx + c) + a.xb[c];
}

// ----------------------------------------------------------------------------- gates ----
// Any sizes: one block per (16 tokens, block of channels), a channel per thread.
constexpr int LG_TOK = 16;
template <class T>
__global__ void __launch_bounds__(128) k_lru_gates_any(LruArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  constexpr int KT = 64;
  __shared__ float su[LG_TOK][KT];
  const int n = a.W / a.blocks, c0 = blockIdx.y * n;
  const int64_t m0 = (int64_t)blockIdx.x * LG_TOK;
  const int tokens = (int)min((int64_t)LG_TOK, a.rows.M - m0);
  for (int e0 = 0; e0 < n; e0 += 128) {
    const int e = e0 + threadIdx.x, c = c0 + e;
    float zr[LG_TOK], zi[LG_TOK];
#pragma unroll
    for (int t = 0; t < LG_TOK; ++t) zr[t] = zi[t] = 0.f;
    for (int k0 = 0; k0 < n; k0 += KT) {
      __syncthreads();
      for (int i = threadIdx.x; i < LG_TOK * KT; i += 128) {
        const int t = i / KT, k = i - t * KT;
        su[t][k] = t < tokens && k0 + k < n ? ld((const T*)a.u + (m0 + t) * a.W + c0 + k0 + k) : 0.f;
      }
      __syncthreads();
      if (e < n)
        for (int k = 0; k < min(KT, n - k0); ++k) {
          const float wr = ld((const T*)a.ra + (int64_t)c * n + k0 + k), wi = ld((const T*)a.ri + (int64_t)c * n + k0 + k);
#pragma unroll
          for (int t = 0; t < LG_TOK; ++t) { zr[t] += wr * su[t][k]; zi[t] += wi * su[t][k]; }
        }
    }
    if (e < n)
#pragma unroll
      for (int t = 0; t < LG_TOK; ++t)
        if (t < tokens) {
          const int64_t o = (m0 + t) * a.W + c;
          const float2 g = gate_pair(zr[t] + a.ra_b[c], zi[t] + a.ri_b[c], a.f[c], ld((const T*)a.u + o));
          a.a[o] = g.x;
          a.b[o] = g.y;
        }
  }
}

// Blocks of a multiple of 16 channels: 64 tokens x 64 output channels of both gates, 64 input channels at a
// time through two buffers.  Products of bf16 values, exact, summed in f32.
constexpr int LG_LD = 72;
__global__ void __launch_bounds__(256) k_lru_gates(LruArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr uint32_t TILE = 64 * LG_LD * 2;
  const uint32_t base = (uint32_t)__cvta_generic_to_shared(smem);
  const int n = a.W / a.blocks, per = (n + 63) / 64;
  const int blk = blockIdx.y / per, e0 = (blockIdx.y - blk * per) * 64;
  const int64_t m0 = (int64_t)blockIdx.x * 64;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wm = warp & 3, wn = warp >> 2;
  const int nk = (n + 63) / 64;
  const __nv_bfloat16* u = (const __nv_bfloat16*)a.u;
  auto load = [&](int kt) {
    const uint32_t b = base + (uint32_t)(kt & 1) * 3 * TILE;
    for (int i = tid; i < 64 * 8; i += 256) {
      const int r = i >> 3, k = kt * 64 + (i & 7) * 8;
      const uint32_t d = (uint32_t)(r * LG_LD + (i & 7) * 8) * 2u;
      const bool ok = k < n, tok = ok && m0 + r < a.rows.M, out = ok && e0 + r < n;
      cp_async16(b + d, u + (tok ? (m0 + r) * a.W + blk * n + k : 0), tok ? 16 : 0);
      const int64_t w = out ? (int64_t)(blk * n + e0 + r) * n + k : 0;
      cp_async16(b + TILE + d, (const __nv_bfloat16*)a.ra + w, out ? 16 : 0);
      cp_async16(b + 2 * TILE + d, (const __nv_bfloat16*)a.ri + w, out ? 16 : 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float acc[2][4][4];
#pragma unroll
  for (int g = 0; g < 2; ++g)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[g][j][0] = acc[g][j][1] = acc[g][j][2] = acc[g][j][3] = 0.f;
  load(0);
  for (int kt = 0; kt < nk; ++kt) {
    if (kt + 1 < nk) {
      load(kt + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const uint32_t b = base + (uint32_t)(kt & 1) * 3 * TILE;
#pragma unroll
    for (int kk = 0; kk < 64; kk += 16) {
      uint32_t fa[4];
      const int r = wm * 16 + (lane & 7) + 8 * ((lane >> 3) & 1), c = kk + 8 * (lane >> 4);
      ldsm_x4(b + (uint32_t)(r * LG_LD + c) * 2u, fa[0], fa[1], fa[2], fa[3]);
#pragma unroll
      for (int g = 0; g < 2; ++g)
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          uint32_t fb[4];
          const int rn = wn * 32 + j * 8 + (lane & 7) + 8 * (lane >> 4), ck = kk + 8 * ((lane >> 3) & 1);
          ldsm_x4(b + (uint32_t)(1 + g) * TILE + (uint32_t)(rn * LG_LD + ck) * 2u, fb[0], fb[1], fb[2], fb[3]);
          mma_bf16(acc[g][j], fa[0], fa[1], fa[2], fa[3], fb[0], fb[1]);
          mma_bf16(acc[g][j + 1], fa[0], fa[1], fa[2], fa[3], fb[2], fb[3]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int e = e0 + wn * 32 + j * 8 + (lane & 3) * 2, c = blk * n + e;
    if (e >= n) continue;  // (n is a multiple of 16: both columns exist or neither)
    const float2 br = *(const float2*)(a.ra_b + c), bi = *(const float2*)(a.ri_b + c), f = *(const float2*)(a.f + c);
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int64_t m = m0 + wm * 16 + (lane >> 2) + 8 * x;
      if (m >= a.rows.M) continue;
      const float2 uu = __bfloat1622float2(*(const __nv_bfloat162*)(u + m * a.W + c));
      const float2 g0 = gate_pair_fast(acc[0][j][2 * x] + br.x, acc[1][j][2 * x] + bi.x, f.x, uu.x);
      const float2 g1 = gate_pair_fast(acc[0][j][2 * x + 1] + br.y, acc[1][j][2 * x + 1] + bi.y, f.y, uu.y);
      *(float2*)(a.a + m * a.W + c) = make_float2(g0.x, g1.x);
      *(float2*)(a.b + m * a.W + c) = make_float2(g0.y, g1.y);
    }
  }
}

// ------------------------------------------------------------------------------ scan ----
// One block per (32 channels, row): a tile of 128 tokens at a time, 8 per warp.  A segment's tokens compose to
// S -> A S + B; the 16 segments of a channel are chained through shared memory.
constexpr int LS_SEG = 16, LS_TOK = 8, LS_TILE = LS_SEG * LS_TOK;
template <class TP, class T>
__global__ void __launch_bounds__(32 * LS_SEG) k_lru_scan(LruArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __shared__ float sA[2][LS_SEG][32], sB[2][LS_SEG][32];
  const int lane = threadIdx.x & 31, seg = threadIdx.x >> 5;
  const int c = blockIdx.x * 32 + lane, row = blockIdx.y;
  const bool live = c < a.W;
  const int64_t s0 = a.rows.start[row];
  const int len = (int)(a.rows.start[row + 1] - s0);
  float* Sg = a.S + (int64_t)a.rows.slot[row] * a.W + c;
  float S = live && row_pos0(a.rows, row) > 0 ? *Sg : 0.f;  // before the tile: the same in every segment
  const float yb = live ? a.yb[c] : 0.f;
  float av[LS_TOK], bv[LS_TOK], yv[LS_TOK];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int k = 0; k < LS_TOK; ++k) {
      const int t = t0 + seg * LS_TOK + k;
      const bool in = live && t < len;
      const int64_t m = s0 + (in ? t : 0);
      av[k] = in ? a.a[m * a.W + c] : 1.f;
      bv[k] = in ? a.b[m * a.W + c] : 0.f;
      yv[k] = in ? ld((const TP*)a.y + m * a.ldx + c) : 0.f;
    }
  };
  fetch(0);
  for (int t0 = 0, p = 0; t0 < len; t0 += LS_TILE, p ^= 1) {
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int k = 0; k < LS_TOK; ++k) {
      A *= av[k];
      B = av[k] * B + bv[k];
    }
    sA[p][seg][lane] = A;
    sB[p][seg][lane] = B;
    __syncthreads();
    float mine = S;  // before this segment
    for (int s = 0; s < LS_SEG; ++s) {
      if (s == seg) mine = S;
      S = sA[p][s][lane] * S + sB[p][s][lane];
    }
    float out[LS_TOK];
#pragma unroll
    for (int k = 0; k < LS_TOK; ++k) {
      mine = av[k] * mine + bv[k];
      out[k] = mine * (sizeof(TP) == 2 ? gelu_fast(yv[k] + yb) : gelu_exact(yv[k] + yb));
    }
    if (t0 + LS_TILE < len) fetch(t0 + LS_TILE);
#pragma unroll
    for (int k = 0; k < LS_TOK; ++k) {
      const int t = t0 + seg * LS_TOK + k;
      if (live && t < len) st((T*)a.out + (s0 + t) * a.ld_out + c, out[k]);
    }
  }
  if (live && seg == 0) *Sg = S;
}

// ----------------------------------------------------------------- one token per row ----
// One block per (block of channels, 32 of its outputs, 8 rows): the convolution of the whole block of every
// row in shared memory, a warp per 4 outputs of both gates, lanes over the inputs; the sums over the lanes
// leave lane l with output l / 8 of row l % 8.  The first weights are requested before the wait.
constexpr int LD_OUT = 32, LD_ROWS = 8;
template <class T>
__device__ __forceinline__ void load4(const T* p, bool in, float* v) {
  if constexpr (sizeof(T) == 2) {
    widen4(in ? *(const uint2*)p : make_uint2(0, 0), v);
  } else {
    const float4 f = in ? *(const float4*)p : make_float4(0.f, 0.f, 0.f, 0.f);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  }
}
// VEC: blocks of a multiple of 4 channels
template <class T, bool VEC>
__global__ void __launch_bounds__(256) k_lru_decode(LruArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  extern __shared__ __align__(16) float su[];  // [LD_ROWS][np], np = n rounded up to 128
  const int n = a.W / a.blocks, np = (n + 127) / 128 * 128, per = (n + LD_OUT - 1) / LD_OUT;
  const int blk = blockIdx.x / per, e0 = (blockIdx.x - blk * per) * LD_OUT, r0 = blockIdx.y * LD_ROWS;
  const int rows = min(LD_ROWS, a.rows.rows - r0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int o0 = e0 + warp * 4;                     // this warp's outputs inside the block
  float w[2][4][4];                                 // [gate][output][input]
  auto weights = [&](int k) {
#pragma unroll
    for (int o = 0; o < 4; ++o) {
      const bool in = o0 + o < n && k < n;
      const int64_t at = in ? (int64_t)(blk * n + o0 + o) * n + k : 0;
#pragma unroll
      for (int g = 0; g < 2; ++g) {
        const T* p = (const T*)(g ? a.ri : a.ra) + at;
        if constexpr (VEC) load4(p, in, w[g][o]);
        else
#pragma unroll
          for (int e = 0; e < 4; ++e) w[g][o][e] = in && k + e < n ? ld(p + e) : 0.f;
      }
    }
  };
  weights(4 * lane);
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const float* x = (const float*)a.x;
  for (int i = tid; i < LD_ROWS * np; i += 256) {
    const int q = i / np, e = i - q * np, c = blk * n + e, row = r0 + q;
    float v = 0.f;
    if (q < rows && e < n) {
      const int64_t pos = row_pos0(a.rows, row);
      float* tail = a.tail + (int64_t)a.rows.slot[row] * a.taps * a.W;
      const int ring = (int)((uint32_t)pos % (uint32_t)a.taps);
      const float now = x[(int64_t)row * a.ldx + c] + a.xb[c];
      v = a.conv_b[c] + a.conv_w[(int64_t)c * a.taps + a.taps - 1] * now;
      for (int j = 1; j < a.taps; ++j)
        if (pos >= j) v += a.conv_w[(int64_t)c * a.taps + a.taps - 1 - j] * tail[(int64_t)(ring >= j ? ring - j : ring - j + a.taps) * a.W + c];
      if (e >= e0 && e < e0 + LD_OUT) tail[(int64_t)ring * a.W + c] = now;  // read by no block of this step
      v = as(v, (const T*)nullptr);
    }
    su[i] = v;
  }
  __syncthreads();
  if (o0 >= n) return;
  float z[64];  // [output][row][gate]
#pragma unroll
  for (int i = 0; i < 64; ++i) z[i] = 0.f;
  for (int k0 = 0; k0 < n; k0 += 128) {
    if (k0) weights(k0 + 4 * lane);
#pragma unroll
    for (int q = 0; q < LD_ROWS; ++q) {
      const float4 u = *(const float4*)(su + q * np + k0 + 4 * lane);
#pragma unroll
      for (int o = 0; o < 4; ++o)
#pragma unroll
        for (int g = 0; g < 2; ++g)
          z[(o * 8 + q) * 2 + g] += w[g][o][0] * u.x + w[g][o][1] * u.y + w[g][o][2] * u.z + w[g][o][3] * u.w;
    }
  }
#pragma unroll
  for (int step = 0; step < 5; ++step) {
    const int off = 16 >> step, half = 32 >> step;  // values kept: half, the upper ones by lanes with this bit
    const bool upper = lane & off;
#pragma unroll
    for (int i = 0; i < 32; ++i)
      if (i < half) {
        const float send = upper ? z[i] : z[i + half], keep = upper ? z[i + half] : z[i];
        z[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
      }
  }
  const int e = o0 + (lane >> 3), q = lane & 7, c = blk * n + e;
  if (e < n && q < rows) {
    const int row = r0 + q;
    float* Sg = a.S + (int64_t)a.rows.slot[row] * a.W + c;
    const float2 g = gate_pair(z[0] + a.ra_b[c], z[1] + a.ri_b[c], a.f[c], su[q * np + e]);
    const float S = g.x * (row_pos0(a.rows, row) > 0 ? *Sg : 0.f) + g.y;
    *Sg = S;
    st((T*)a.out + (int64_t)row * a.ld_out + c, S * gelu_exact(((const float*)a.y)[(int64_t)row * a.ldx + c] + a.yb[c]));
  }
}

}  // namespace

// one token per row, f32 projections
int k_launch_lru_decode(cg_ctx* c, const LruArgs& a) {
  if (a.rows.rows == 0) return CG_OK;
  const int n = a.W / a.blocks;
  const size_t smem = (size_t)LD_ROWS * ((n + 127) / 128 * 128) * 4;
  if (smem > 200 * 1024) return fail(c, CG_ERR_UNSUPPORTED, "recurrence: gate blocks too wide");
  const bool vec = n % 4 == 0;
  auto kernel = a.out_bf16 ? (vec ? k_lru_decode<__nv_bfloat16, true> : k_lru_decode<__nv_bfloat16, false>)
                           : (vec ? k_lru_decode<float, true> : k_lru_decode<float, false>);
  static PerDeviceSize configured_on[4];
  size_t& configured = configured_on[2 * (a.out_bf16 ? 1 : 0) + (vec ? 1 : 0)].at(c->core->device);
  if (smem > 48 * 1024 && smem > configured) {
    CG_CUDA(c, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = smem;
  }
  dim3 grid((unsigned)(a.blocks * ((n + LD_OUT - 1) / LD_OUT)), (unsigned)((a.rows.rows + LD_ROWS - 1) / LD_ROWS));
  CG_CUDA(c, launch_kernel(c, kernel, grid, dim3(256), smem, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_lru_prompt(cg_ctx* c, const LruArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  const int n = a.W / a.blocks;
  const dim3 conv_grid((unsigned)((a.rows.M + LC_TOK - 1) / LC_TOK), (unsigned)((a.W + 127) / 128));
  if (a.in_bf16 && a.W % 4 == 0 && a.taps <= 4) {
    const dim3 grid((unsigned)(a.n_chunks * (RECUR_CHUNK / LV_TOK)), (unsigned)((a.W + 511) / 512));
    auto conv = a.taps == 1 ? k_lru_conv_vec<1> : a.taps == 2 ? k_lru_conv_vec<2> : a.taps == 3 ? k_lru_conv_vec<3> : k_lru_conv_vec<4>;
    CG_CUDA(c, launch_kernel(c, conv, grid, dim3(128), 0, 1, a));
  } else {
    auto conv = !a.out_bf16 ? k_lru_conv<float, float> : a.in_bf16 ? k_lru_conv<__nv_bfloat16, __nv_bfloat16> : k_lru_conv<float, __nv_bfloat16>;
    CG_CUDA(c, launch_kernel(c, conv, conv_grid, dim3(128), 0, 1, a));
  }
  CG_LAUNCHED(c);
  if (a.taps > 1) {
    auto tail = a.in_bf16 ? k_lru_tail<__nv_bfloat16> : k_lru_tail<float>;
    CG_CUDA(c, launch_kernel(c, tail, dim3((unsigned)((a.W + 127) / 128), (unsigned)a.rows.rows), dim3(128), 0, 1, a));
    CG_LAUNCHED(c);
  }
  if (a.out_bf16 && n % 16 == 0) {
    constexpr size_t smem = (size_t)6 * 64 * LG_LD * 2;
    static PerDeviceFlag configured_on;
    bool& configured = configured_on.at(c->core->device);
    if (!configured) {
      CG_CUDA(c, cudaFuncSetAttribute(k_lru_gates, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
      configured = true;
    }
    const dim3 grid((unsigned)((a.rows.M + 63) / 64), (unsigned)(a.blocks * ((n + 63) / 64)));
    CG_CUDA(c, launch_kernel(c, k_lru_gates, grid, dim3(256), smem, 1, a));
  } else {
    auto gates = a.out_bf16 ? k_lru_gates_any<__nv_bfloat16> : k_lru_gates_any<float>;
    CG_CUDA(c, launch_kernel(c, gates, dim3((unsigned)((a.rows.M + LG_TOK - 1) / LG_TOK), (unsigned)a.blocks), dim3(128), 0, 1, a));
  }
  CG_LAUNCHED(c);
  auto scan = !a.out_bf16 ? k_lru_scan<float, float> : a.in_bf16 ? k_lru_scan<__nv_bfloat16, __nv_bfloat16> : k_lru_scan<float, __nv_bfloat16>;
  CG_CUDA(c, launch_kernel(c, scan, dim3((unsigned)((a.W + 31) / 32), (unsigned)a.rows.rows), dim3(32 * LS_SEG), 0, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace cg
