// recurrent.cu — layers whose memory is a matrix per head: the gated delta rule and the Mamba-2
// state space, both behind short causal convolutions, lightning attention, and the delta rule and gated
// linear attention with a decay per key channel.  State, decays, step sizes, unit norms and
// gates are f32.
#include <algorithm>

#include "act.cuh"
#include "mixers.h"
#include "mma.cuh"

namespace cg {

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float block_sum(float v, float* sh) {
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) sh[wid] = v;
  __syncthreads();
  v = lane < nw ? sh[lane] : 0.f;
  return warp_sum(v);
}
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// The convolution at channel c of token m: the row's place i, its first position p0.
__device__ __forceinline__ float conv_at(const RecurArgs& a, int64_t m, int i, int64_t p0, int c, const float* tail) {
  float v = a.conv_b ? a.conv_b[c] : 0.f;
  if (a.taps == 0) v = a.proj[m * a.ldp + c];
  for (int j = 0; j < a.taps; ++j) {
    float x = 0.f;
    if (j <= i) x = a.proj[(m - j) * a.ldp + c];
    else if (p0 + i - j >= 0) x = tail[(int64_t)((p0 + i - j) % a.taps) * a.C + c];
    v += a.conv_w[(int64_t)c * a.taps + a.taps - 1 - j] * x;
  }
  return a.linear ? v : silu(v);
}

// One block per token, one warp per unit: a query head, a key head, or 128 other channels.
__global__ void __launch_bounds__(256) k_conv_heads(RecurArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int64_t m = blockIdx.x;
  const int row = a.rows.tok_row[m];
  const int i = (int)(m - a.rows.start[row]);
  const int64_t p0 = row_pos0(a.rows, row);
  const float* tail = a.tail + (int64_t)a.rows.slot[row] * a.taps * a.C;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  float* out = a.cv + m * a.ldc;
  const int norm_units = a.delta ? 2 * a.KH : 0;          // delta: q heads then k heads, contiguous from column 0
  const int c_rest = norm_units * a.dk;
  const int units = norm_units + (a.C - c_rest + 127) / 128;
  for (int u = warp; u < units; u += nw) {
    if (u < norm_units) {
      const int c0 = u * a.dk;
      float ss = 0.f;
      for (int e = lane; e < a.dk; e += 32) {
        const float v = conv_at(a, m, i, p0, c0 + e, tail);
        out[c0 + e] = v;
        ss += v * v;
      }
      ss = warp_sum(ss);
      float f = 1.f / sqrtf(ss + 1e-6f);
      if (u < a.KH) f *= 1.f / sqrtf((float)a.dk);
      for (int e = lane; e < a.dk; e += 32) out[c0 + e] *= f;  // this lane's own stores
    } else {
      const int c0 = c_rest + (u - norm_units) * 128;
      for (int e = lane; e < 128 && c0 + e < a.C; e += 32)
        out[c0 + e] = conv_at(a, m, i, p0, c0 + e, tail) * (a.q_scale != 1.f && c0 + e < a.k_off ? a.q_scale : 1.f);
    }
  }
  const float* sp = a.proj + m * a.ldp + a.small_off;
  for (int h = threadIdx.x; h < a.H; h += blockDim.x) {
    if (a.key_decay) {
      a.co[m * a.H + h] = a.delta ? 1.f / (1.f + expf(-sp[h])) : 1.f;
      continue;
    }
    if (a.log_decay) {
      a.gl[m * a.H + h] = a.log_decay[h];
      a.co[m * a.H + h] = 1.f;
      continue;
    }
    const float dt = softplus(sp[a.delta ? a.H + h : h] + a.dt_bias[h]);
    a.gl[m * a.H + h] = -expf(a.a_log[h]) * dt;
    a.co[m * a.H + h] = a.delta ? 1.f / (1.f + expf(-sp[h])) : dt;
  }
}

// the last inputs of the convolution, at their position modulo taps
__global__ void k_conv_tail(RecurArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int row = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= a.C) return;
  const int64_t s0 = a.rows.start[row], p0 = row_pos0(a.rows, row);
  const int len = (int)(a.rows.start[row + 1] - s0);
  float* tail = a.tail + (int64_t)a.rows.slot[row] * a.taps * a.C;
  for (int i = max(0, len - a.taps + 1); i < len; ++i) tail[(int64_t)((p0 + i) % a.taps) * a.C + c] = a.proj[(s0 + i) * a.ldp + c];
}

// One block per (128 columns, token): the row of x in shared memory, a column per thread.
__global__ void __launch_bounds__(128) k_low_rank(LowRank a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  extern __shared__ float sx[];
  const int64_t m = blockIdx.x;
  const int n = blockIdx.y * 128 + threadIdx.x;
  for (int j = threadIdx.x; j < a.R; j += 128) sx[j] = a.x[m * a.ldx + j];
  __syncthreads();
  if (n >= a.N) return;
  float v = 0.f;
  for (int j = 0; j < a.R; ++j)
    v += sx[j] * (a.w_bf16 ? __bfloat162float(((const __nv_bfloat16*)a.w)[(int64_t)n * a.R + j]) : ((const float*)a.w)[(int64_t)n * a.R + j]);
  if (a.coef) v = -a.coef[n / a.zs] * softplus(a.sign * (v + a.bias[n]));
  a.out[m * a.N + n] = v;
}

// One block per (32 value columns, head, row), token by token.  Four threads share a column, each
// with every fourth key row of it; the state's columns live in shared memory.
__global__ void __launch_bounds__(128) k_recur_steps(RecurArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  extern __shared__ float sm[];
  float* S = sm;                     // [dk][32]
  float* ks = S + a.dk * 32;         // [dk]
  float* qs = ks + a.dk;             // [dk]
  float* gs = qs + a.dk;             // [dk] decays
  float* red = gs + a.dk;            // [4][32]
  const int row = blockIdx.z, h = blockIdx.y, e0 = blockIdx.x * 32;
  const int tid = threadIdx.x, col = tid & 31, part = tid >> 5;
  const int e = e0 + col;
  const bool live = e < a.dv;
  const int64_t s0 = a.rows.start[row];
  const int len = (int)(a.rows.start[row + 1] - s0);
  float* Sg = a.S + ((int64_t)a.rows.slot[row] * a.H + h) * a.dk * a.dvs;
  const bool first = row_pos0(a.rows, row) == 0;
  for (int i = part; i < a.dk; i += 4) S[i * 32 + col] = live && !first ? Sg[(int64_t)i * a.dvs + e] : 0.f;
  const int kh = h / (a.H / a.KH);
  for (int t = 0; t < len; ++t) {
    const int64_t m = s0 + t;
    const float* cv = a.cv + m * a.ldc;
    __syncthreads();
    for (int i = tid; i < a.dk; i += 128) {
      ks[i] = cv[a.k_off + kh * a.qs + i];
      qs[i] = cv[a.q_off + kh * a.qs + i];
      gs[i] = expf(a.key_decay ? a.gl[m * (int64_t)a.H * a.zs + h * a.zs + i] : a.gl[m * a.H + h]);
    }
    const float v = live ? cv[a.v_off + h * a.vs + e] : 0.f;
    const float co = a.co[m * a.H + h];
    __syncthreads();
    float u = co * v;
    if (a.delta) {
      float p = 0.f;
      for (int i = part; i < a.dk; i += 4) {
        const float x = gs[i] * S[i * 32 + col];
        S[i * 32 + col] = x;
        p += x * ks[i];
      }
      red[part * 32 + col] = p;
      __syncthreads();
      u = co * (v - ((red[col] + red[32 + col]) + (red[64 + col] + red[96 + col])));
      __syncthreads();
    }
    float o = 0.f;
    for (int i = part; i < a.dk; i += 4) {
      const float x = (a.delta ? S[i * 32 + col] : gs[i] * S[i * 32 + col]) + ks[i] * u;
      S[i * 32 + col] = x;
      o += x * qs[i];
    }
    red[part * 32 + col] = o;
    __syncthreads();
    if (part == 0 && live) {
      o = (red[col] + red[32 + col]) + (red[64 + col] + red[96 + col]);
      if (a.dskip) o += a.dskip[h] * v;
      a.o[m * (int64_t)a.H * a.dvs + h * a.dvs + e] = o;
    }
  }
  if (live)
    for (int i = part; i < a.dk; i += 4) Sg[(int64_t)i * a.dvs + e] = S[i * 32 + col];
}

// ------------------------------------------------------------------ one token per row ----
// One block per (head, row).  A thread keeps four columns of up to RD_ROWS rows of the state in
// registers from the load to the store; sums over the key dimension go through shared memory.
// KD: a decay per key channel; the second factors of the low-rank projections are applied here, a row of them
// per thread, from shared memory where they fit (rows R + 8 apart: no bank conflicts).
__device__ __forceinline__ float low_rank_staged(const float* x, const __nv_bfloat16* w, int R) {
  float v[2] = {0.f, 0.f};
#pragma unroll 2
  for (int j = 0; j < R; j += 8) {
    const uint4 r = *(const uint4*)(w + j);
    const float4 x0 = *(const float4*)(x + j), x1 = *(const float4*)(x + j + 4);
    v[0] += x0.x * __uint_as_float(r.x << 16) + x0.y * __uint_as_float(r.x & 0xffff0000u);
    v[1] += x0.z * __uint_as_float(r.y << 16) + x0.w * __uint_as_float(r.y & 0xffff0000u);
    v[0] += x1.x * __uint_as_float(r.z << 16) + x1.y * __uint_as_float(r.z & 0xffff0000u);
    v[1] += x1.z * __uint_as_float(r.w << 16) + x1.w * __uint_as_float(r.w & 0xffff0000u);
  }
  return v[0] + v[1];
}
template <int RD_ROWS, bool KD>
__global__ void __launch_bounds__(256, RD_ROWS <= 8 ? 3 : 2) k_recur_decode(RecurArgs a, GatedNorm n) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  __shared__ float sq[128], sk[128], sv[128], so[128], sg[4];
  __shared__ float sd[KD ? 128 : 1], sgate[KD ? 128 : 1];  // decays, gates before their activation
  // KD: [a_rank], [g_rank]; with w_staged then this head's rows of the second factors
  extern __shared__ __align__(16) float low[];
  __nv_bfloat16* const staged = (__nv_bfloat16*)(low + (a.a_rank + a.g_rank));  // (ranks are multiples of 8)
  if (KD && a.w_staged) {
    // weights: on their way while the projection still runs
    const uint32_t to = (uint32_t)__cvta_generic_to_shared(staged);
    const int na = a.dk * a.a_rank / 8, ng = a.w_g2 ? a.dv * a.g_rank / 8 : 0;
    const __nv_bfloat16* wa = (const __nv_bfloat16*)a.w_a2 + (int64_t)blockIdx.x * a.zs * a.a_rank;
    const __nv_bfloat16* wg = (const __nv_bfloat16*)a.w_g2 + (int64_t)blockIdx.x * a.dv * a.g_rank;
    for (int i = threadIdx.x; i < na + ng; i += 256) {
      const bool decay = i < na;
      const int R8 = (decay ? a.a_rank : a.g_rank) / 8, x = decay ? i : i - na, r = x / R8;
      cp_async16(to + (decay ? 0u : (uint32_t)(a.dk * (a.a_rank + 8)) * 2u) + (uint32_t)(r * (8 * R8 + 8) + (x - r * R8) * 8) * 2u,
                 (decay ? wa : wg) + x * 8, 16);
    }
  }
  __shared__ __align__(16) float red[1024];
  const int h = blockIdx.x, row = blockIdx.y, rep = a.H / a.KH, kh = h / rep;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int lpr = a.dvs / 4, rpp = 256 / lpr;         // threads per state row, rows per pass
  const int rg = tid / lpr, cg = tid - rg * lpr;
  const bool act = rg < rpp;
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int64_t m = row, pos = row_pos0(a.rows, row);
  const int slot = a.rows.slot[row];
  float* Sg = a.S + ((int64_t)slot * a.H + h) * a.dk * a.dvs;
  float4 S[RD_ROWS];
#pragma unroll
  for (int i = 0; i < RD_ROWS; ++i) {
    const int r = rg + i * rpp;
    S[i] = act && r < a.dk && pos > 0 ? *(const float4*)(Sg + (int64_t)r * a.dvs + 4 * cg) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  // short convolutions of this head's channels
  const float* p = a.proj + m * a.ldp;
  float* tail = a.tail + (int64_t)slot * a.taps * a.C;
  const int ring = a.taps ? (int)((uint32_t)pos % (uint32_t)a.taps) : 0;  // this position's place among the last inputs
  for (int x = tid; x < 2 * a.dk + a.dvs; x += 256) {
    const int seg = x < a.dk ? 0 : x < 2 * a.dk ? 1 : 2;
    const int e = seg == 0 ? x : seg == 1 ? x - a.dk : x - 2 * a.dk;
    if (seg == 2 && e >= a.dv) { sv[e] = 0.f; continue; }
    const int c = seg == 0 ? a.q_off + kh * a.qs + e : seg == 1 ? a.k_off + kh * a.qs + e : a.v_off + h * a.vs + e;
    const float now = p[c];
    float v = now;
    if (a.taps) {
      v = (a.conv_b ? a.conv_b[c] : 0.f) + a.conv_w[(int64_t)c * a.taps + a.taps - 1] * now;
      for (int j = 1; j < a.taps; ++j)
        if (pos >= j) v += a.conv_w[(int64_t)c * a.taps + a.taps - 1 - j] * tail[(int64_t)(ring >= j ? ring - j : ring - j + a.taps) * a.C + c];
      if (seg == 2 || h % rep == 0) tail[(int64_t)ring * a.C + c] = now;  // read by no block of this step
    }
    if (a.linear) v *= seg == 0 ? a.q_scale : 1.f;
    else v = silu(v);
    (seg == 0 ? sq : seg == 1 ? sk : sv)[e] = v;
  }
  if (KD) {
    for (int j = tid; j < a.a_rank; j += 256) low[j] = p[a.a1_off + j];
    if (a.w_g2)
      for (int j = tid; j < a.g_rank; j += 256) low[a.a_rank + j] = p[a.g1_off + j];
    cp_async_wait_all();
    __syncthreads();
#pragma unroll 1
    for (int e = tid; e < a.dk + a.dv; e += 256) {
      const bool decay = e < a.dk;
      const int64_t r = decay ? (int64_t)h * a.zs + e : (int64_t)h * a.dv + e - a.dk;
      const int R = decay ? a.a_rank : a.g_rank;
      const float* x = decay ? low : low + a.a_rank;
      float v = 0.f;
      if (!decay && !a.w_g2) {
        v = ((const float*)n.gate)[m * n.ldg + r];
      } else if (a.w_staged) {
        v = low_rank_staged(x, staged + (decay ? e * (R + 8) : a.dk * (a.a_rank + 8) + (e - a.dk) * (R + 8)), R);
      } else {
        const void* w = decay ? a.w_a2 : a.w_g2;
#pragma unroll 1
        for (int j = 0; j < R; ++j) v += x[j] * (a.w_bf16 ? __bfloat162float(((const __nv_bfloat16*)w)[r * R + j]) : ((const float*)w)[r * R + j]);
      }
      if (decay) sd[e] = expf(-a.coef[h] * softplus(a.z_sign * (v + a.z_bias[r])));
      else sgate[e - a.dk] = v;
    }
  }
  const float* sp = p + a.small_off;
  if (tid == 64) {
    if (KD) {
      sg[1] = a.delta ? 1.f / (1.f + expf(-sp[h])) : 1.f;
    } else if (a.log_decay) {
      sg[0] = expf(a.log_decay[h]);
      sg[1] = 1.f;
    } else {
      const float dt = softplus(sp[a.delta ? a.H + h : h] + a.dt_bias[h]);
      sg[0] = expf(-expf(a.a_log[h]) * dt);
      sg[1] = a.delta ? 1.f / (1.f + expf(-sp[h])) : dt;
    }
  }
  __syncthreads();
  if (a.delta) {
    if (warp < 2) {
      float* x = warp ? sk : sq;
      float ss = 0.f;
      for (int e = lane; e < a.dk; e += 32) ss += x[e] * x[e];
      ss = warp_sum(ss);
      const float f = (warp ? 1.f : 1.f / sqrtf((float)a.dk)) / sqrtf(ss + 1e-6f);
      for (int e = lane; e < a.dk; e += 32) x[e] *= f;
    }
    __syncthreads();
  }
  const float g0 = sg[0], co = sg[1];
  auto decay = [&](int r) { return KD ? sd[r < a.dk ? r : 0] : g0; };
  auto sum_rows = [&](float4 v) {   // over all rows of the state, for this thread's columns
    if (act) *(float4*)(red + rg * a.dvs + 4 * cg) = v;
    __syncthreads();
    float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
    if (act)
      for (int i = 0; i < rpp; ++i) {
        const float4 r = *(const float4*)(red + i * a.dvs + 4 * cg);
        t.x += r.x; t.y += r.y; t.z += r.z; t.w += r.w;
      }
    return t;
  };
  float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
  if (act) u = *(const float4*)(sv + 4 * cg);
  const float4 v4 = u;
  if (a.delta) {
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < RD_ROWS; ++i) {
      const int r = rg + i * rpp;
      const float k = act && r < a.dk ? sk[r] : 0.f, g = decay(r);
      S[i].x *= g; S[i].y *= g; S[i].z *= g; S[i].w *= g;
      s.x += S[i].x * k; s.y += S[i].y * k; s.z += S[i].z * k; s.w += S[i].w * k;
    }
    s = sum_rows(s);
    u.x -= s.x; u.y -= s.y; u.z -= s.z; u.w -= s.w;
    __syncthreads();
  }
  u.x *= co; u.y *= co; u.z *= co; u.w *= co;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < RD_ROWS; ++i) {
    const int r = rg + i * rpp;
    if (act && r < a.dk) {
      const float k = sk[r], q = sq[r], g = decay(r);
      if (a.delta) {
        S[i].x += k * u.x; S[i].y += k * u.y; S[i].z += k * u.z; S[i].w += k * u.w;
      } else {
        S[i].x = g * S[i].x + k * u.x; S[i].y = g * S[i].y + k * u.y;
        S[i].z = g * S[i].z + k * u.z; S[i].w = g * S[i].w + k * u.w;
      }
      o.x += S[i].x * q; o.y += S[i].y * q; o.z += S[i].z * q; o.w += S[i].w * q;
      *(float4*)(Sg + (int64_t)r * a.dvs + 4 * cg) = S[i];
    }
  }
  o = sum_rows(o);
  if (!a.delta && !KD) {
    if (rg == 0) {
      const float d = a.dskip ? a.dskip[h] : 0.f;
      *(float4*)(a.o + m * (int64_t)a.H * a.dvs + (int64_t)h * a.dvs + 4 * cg) =
          make_float4(o.x + d * v4.x, o.y + d * v4.y, o.z + d * v4.z, o.w + d * v4.w);
    }
    return;
  }
  if (rg == 0) *(float4*)(so + 4 * cg) = o;
  __syncthreads();
  const float* gate = (const float*)n.gate + m * n.ldg + (int64_t)h * a.dv;
  const float x = tid < a.dv ? so[tid] : 0.f;
  const float ss = block_sum(x * x, red);
  if (tid < a.dv) {
    const float z = KD ? sgate[tid] : gate[tid];
    const float y = x / sqrtf(ss / (float)a.dv + n.eps) * n.norm[tid] * (n.sigmoid ? 1.f / (1.f + expf(-z)) : silu(z));
    const int64_t at = m * n.ld_att + (int64_t)h * a.dv + tid;
    if (n.att_bf16) ((__nv_bfloat16*)n.att)[at] = __float2bfloat16_rn(y);
    else ((float*)n.att)[at] = y;
  }
}

// ------------------------------------------------------------------------- gated norm ----
__device__ __forceinline__ float ldg1(const float* p) { return *p; }
__device__ __forceinline__ float ldg1(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ float4 ldg4(const float* p) { return *(const float4*)p; }
__device__ __forceinline__ float4 ldg4(const __nv_bfloat16* p) {
  const uint2 r = *(const uint2*)p;
  const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&r.x), b = __bfloat1622float2(*(const __nv_bfloat162*)&r.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4(float* p, float4 v) { *(float4*)p = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *(uint2*)p = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
}

__device__ __forceinline__ float gate_act(const GatedNorm& a, float x) { return a.sigmoid ? 1.f / (1.f + expf(-x)) : silu(x); }

// One block per (norm group, token), any sizes.
template <class TG, class T>
__global__ void k_gated_norm(GatedNorm a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __shared__ float sh[32];
  const int64_t m = blockIdx.y;
  const int n = a.H * a.dv / a.groups;
  const int c0 = blockIdx.x * n;
  const float* o = a.o + m * (int64_t)a.H * a.dvs;
  const TG* gate = (const TG*)a.gate + m * a.ldg + c0;
  T* out = (T*)a.att + m * a.ld_att + c0;
  auto at = [&](int i) { const int c = c0 + i, h = c / a.dv; return o[h * a.dvs + (c - h * a.dv)]; };
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float v = a.gate_first ? at(i) * gate_act(a, ldg1(gate + i)) : at(i);
    ss += v * v;
  }
  ss = block_sum(ss, sh);
  const float rms = sqrtf(ss / (float)n + a.eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    st(out + i, at(i) * gate_act(a, ldg1(gate + i)) / rms * a.norm[a.shared_gain ? i : c0 + i]);
  }
}

// Groups of whole 128-bit vectors, kept in registers: G threads per group (a warp, or a block).
template <class TG, class T, int V>
__global__ void k_gated_norm_vec(GatedNorm a, int n, int units, int threads) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __shared__ float sh[32];
  const int per = blockDim.x / threads, sub = threadIdx.x / threads, t = threadIdx.x - sub * threads;
  const int64_t unit = blockIdx.x * (int64_t)per + sub;
  const int64_t m = unit / units;
  const int c0 = (int)(unit - m * units) * n;
  const bool live = m < a.M;
  const float* o = a.o + m * (int64_t)a.H * a.dv + c0;
  const TG* gate = (const TG*)a.gate + m * a.ldg + c0;
  T* out = (T*)a.att + m * a.ld_att + c0;
  float4 x[V], g[V];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const int i = 4 * (t + j * threads);
    x[j] = g[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live && i < n) {
      x[j] = *(const float4*)(o + i);
      g[j] = ldg4(gate + i);
    }
  }
#pragma unroll
  for (int j = 0; j < V; ++j) {
    if (a.sigmoid)
      g[j] = sizeof(TG) == 2 ? make_float4(sigmoid_fast(g[j].x), sigmoid_fast(g[j].y), sigmoid_fast(g[j].z), sigmoid_fast(g[j].w))
                             : make_float4(gate_act(a, g[j].x), gate_act(a, g[j].y), gate_act(a, g[j].z), gate_act(a, g[j].w));
    else
      g[j] = sizeof(TG) == 2 ? make_float4(silu_fast(g[j].x), silu_fast(g[j].y), silu_fast(g[j].z), silu_fast(g[j].w))
                             : make_float4(silu(g[j].x), silu(g[j].y), silu(g[j].z), silu(g[j].w));
    if (a.gate_first) { x[j].x *= g[j].x; x[j].y *= g[j].y; x[j].z *= g[j].z; x[j].w *= g[j].w; }
    ss += x[j].x * x[j].x + x[j].y * x[j].y + x[j].z * x[j].z + x[j].w * x[j].w;
  }
  ss = threads == 32 ? warp_sum(ss) : block_sum(ss, sh);
  const float inv = 1.f / sqrtf(ss / (float)n + a.eps);
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const int i = 4 * (t + j * threads);
    if (!live || i >= n) continue;
    const float4 w = *(const float4*)(a.norm + (a.shared_gain ? 0 : c0) + i);
    float4 r = make_float4(x[j].x * inv * w.x, x[j].y * inv * w.y, x[j].z * inv * w.z, x[j].w * inv * w.w);
    if (!a.gate_first) { r.x *= g[j].x; r.y *= g[j].y; r.z *= g[j].z; r.w *= g[j].w; }
    st4(out + i, r);
  }
}

template <class TG, class T>
int launch_gated_norm(cg_ctx* c, const GatedNorm& a) {
  const int units = a.groups;
  const int n = a.H * a.dv / units;
  const bool vec = a.dv == a.dvs && n % 4 == 0 && a.ldg % 4 == 0 && a.ld_att % 4 == 0 && (((uintptr_t)a.gate | (uintptr_t)a.norm) & 15) == 0 && n <= 16384;
  if (vec && n <= 512) {
    const int64_t blocks = (a.M * units + 7) / 8;
    if (n <= 128) CG_CUDA(c, launch_kernel(c, k_gated_norm_vec<TG, T, 1>, dim3((unsigned)blocks), dim3(256), 0, 1, a, n, units, 32));
    else CG_CUDA(c, launch_kernel(c, k_gated_norm_vec<TG, T, 4>, dim3((unsigned)blocks), dim3(256), 0, 1, a, n, units, 32));
  } else if (vec) {
    const int threads = n <= 4096 ? 256 : n <= 8192 ? 512 : 1024;
    CG_CUDA(c, launch_kernel(c, k_gated_norm_vec<TG, T, 4>, dim3((unsigned)(a.M * units)), dim3(threads), 0, 1, a, n, units, threads));
  } else {
    dim3 grid((unsigned)units, (unsigned)a.M);
    if (grid.y > 65535) return fail(c, CG_ERR_UNSUPPORTED, "recurrence: too many tokens in one portion");
    CG_CUDA(c, launch_kernel(c, k_gated_norm<TG, T>, grid, dim3(std::min(512, (n + 31) / 32 * 32)), 0, 1, a));
  }
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace

constexpr size_t LOW_RANK_SMEM = 70 * 1024;  // of a decode block: three share an SM

bool recur_decode_supported(int dk, int dv) { return dk <= 128 && dv <= 128; }

int k_launch_recur_decode(cg_ctx* c, const RecurArgs& a, const GatedNorm& n) {
  if (a.rows.rows == 0) return CG_OK;
  const int rpp = 256 / (a.dvs / 4);  // state rows per pass
  const bool few = (a.dk + rpp - 1) / rpp <= 8;
  auto kernel = a.key_decay ? (few ? k_recur_decode<8, true> : k_recur_decode<16, true>) : few ? k_recur_decode<8, false> : k_recur_decode<16, false>;
  RecurArgs args = a;
  size_t smem = a.key_decay ? (size_t)(a.a_rank + a.g_rank) * 4 : 0;
  if (smem > 32 * 1024) return fail(c, CG_ERR_UNSUPPORTED, "recurrence: low-rank projections too wide");
  if (a.key_decay && a.w_bf16) {
    const size_t rows = ((size_t)a.dk * (a.a_rank + 8) + (a.w_g2 ? (size_t)a.dv * (a.g_rank + 8) : 0)) * 2;
    args.w_staged = a.a_rank % 8 == 0 && a.g_rank % 8 == 0 && smem + rows <= LOW_RANK_SMEM;
    if (args.w_staged) smem += rows;
    static PerDeviceFlag configured_on[2];
    bool& configured = configured_on[few ? 1 : 0].at(c->core->device);
    if (!configured) {
      CG_CUDA(c, cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)LOW_RANK_SMEM));
      configured = true;
    }
  }
  CG_CUDA(c, launch_kernel(c, kernel, dim3((unsigned)a.H, (unsigned)a.rows.rows), dim3(256), smem, 1, args, n));
  CG_LAUNCHED(c);
  return a.delta || a.key_decay ? CG_OK : k_launch_gated_norm(c, n);
}

int k_launch_low_rank(cg_ctx* c, const LowRank& a, int64_t M) {
  if (M == 0) return CG_OK;
  if (a.R > 8192) return fail(c, CG_ERR_UNSUPPORTED, "recurrence: low-rank projections too wide");
  CG_CUDA(c, launch_kernel(c, k_low_rank, dim3((unsigned)M, (unsigned)((a.N + 127) / 128)), dim3(128), (size_t)a.R * 4, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_recur_steps(cg_ctx* c, const RecurArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  CG_CUDA(c, launch_kernel(c, k_conv_heads, dim3((unsigned)a.rows.M), dim3(256), 0, 1, a));
  CG_LAUNCHED(c);
  if (a.taps > 1) {
    CG_CUDA(c, launch_kernel(c, k_conv_tail, dim3((unsigned)((a.C + 127) / 128), (unsigned)a.rows.rows), dim3(128), 0, 1, a));
    CG_LAUNCHED(c);
  }
  const size_t smem = (size_t)(a.dk * 35 + 128) * 4;
  static PerDeviceSize configured_on;
  size_t& configured = configured_on.at(c->core->device);
  if (smem > 48 * 1024 && smem > configured) {
    if (smem > 227 * 1024) return fail(c, CG_ERR_UNSUPPORTED, "recurrence: key size too large");
    CG_CUDA(c, cudaFuncSetAttribute(k_recur_steps, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = smem;
  }
  dim3 grid((unsigned)((a.dv + 31) / 32), (unsigned)a.H, (unsigned)a.rows.rows);
  CG_CUDA(c, launch_kernel(c, k_recur_steps, grid, dim3(128), smem, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_gated_norm(cg_ctx* c, const GatedNorm& a) {
  if (a.M == 0) return CG_OK;
  if (a.gate_bf16) return a.att_bf16 ? launch_gated_norm<__nv_bfloat16, __nv_bfloat16>(c, a) : launch_gated_norm<__nv_bfloat16, float>(c, a);
  return a.att_bf16 ? launch_gated_norm<float, __nv_bfloat16>(c, a) : launch_gated_norm<float, float>(c, a);
}

}  // namespace cg
