// recurrent.cu — layers whose memory is a matrix per head: the gated delta rule and the Mamba-2
// state space, both behind short causal convolutions.  State, decays, step sizes, unit norms and
// gates are f32.
#include <algorithm>

#include "mixers.h"

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

// input of the convolution `back` tokens before token m of its row (i = m's place in the row)
__device__ __forceinline__ float conv_in(const RecurArgs& a, int64_t m, int i, int back, int c, bool first, const float* tail) {
  if (back <= i) return a.proj[(m - back) * a.ldp + c];
  if (first) return 0.f;
  return tail[(int64_t)(a.taps - 1 + i - back) * a.C + c];
}
__device__ __forceinline__ float conv_at(const RecurArgs& a, int64_t m, int i, int c, bool first, const float* tail) {
  float v = a.conv_b ? a.conv_b[c] : 0.f;
  for (int j = 0; j < a.taps; ++j) v += a.conv_w[(int64_t)c * a.taps + a.taps - 1 - j] * conv_in(a, m, i, j, c, first, tail);
  return silu(v);
}

// One block per token, one warp per unit: a query head, a key head, or 128 other channels.
__global__ void __launch_bounds__(256) k_conv_heads(RecurArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int64_t m = blockIdx.x;
  const int row = a.rows.tok_row[m];
  const int i = (int)(m - a.rows.start[row]);
  const bool first = row_pos0(a.rows, row) == 0;
  const float* tail = a.tail + (int64_t)a.rows.slot[row] * (a.taps - 1) * a.C;
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
        const float v = conv_at(a, m, i, c0 + e, first, tail);
        out[c0 + e] = v;
        ss += v * v;
      }
      ss = warp_sum(ss);
      float f = 1.f / sqrtf(ss + 1e-6f);
      if (u < a.KH) f *= 1.f / sqrtf((float)a.dk);
      for (int e = lane; e < a.dk; e += 32) out[c0 + e] *= f;  // this lane's own stores
    } else {
      const int c0 = c_rest + (u - norm_units) * 128;
      for (int e = lane; e < 128 && c0 + e < a.C; e += 32) out[c0 + e] = conv_at(a, m, i, c0 + e, first, tail);
    }
  }
  const float* sp = a.proj + m * a.ldp + a.small_off;
  for (int h = threadIdx.x; h < a.H; h += blockDim.x) {
    const float dt = softplus(sp[a.delta ? a.H + h : h] + a.dt_bias[h]);
    a.gl[m * a.H + h] = -expf(a.a_log[h]) * dt;
    a.co[m * a.H + h] = a.delta ? 1.f / (1.f + expf(-sp[h])) : dt;
  }
}

constexpr int MAX_TAPS = 17;

__global__ void k_conv_tail(RecurArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int row = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= a.C) return;
  const int64_t s0 = a.rows.start[row];
  const int len = (int)(a.rows.start[row + 1] - s0);
  const bool first = row_pos0(a.rows, row) == 0;
  float* tail = a.tail + (int64_t)a.rows.slot[row] * (a.taps - 1) * a.C;
  float v[MAX_TAPS - 1];
  const int n = a.taps - 1;
#pragma unroll
  for (int j = 0; j < MAX_TAPS - 1; ++j) {
    if (j < n) {
      const int off = len - n + j;  // place in the row; negative: before it
      v[j] = off >= 0 ? a.proj[(s0 + off) * a.ldp + c] : (first ? 0.f : tail[(int64_t)(off + n) * a.C + c]);
    }
  }
#pragma unroll
  for (int j = 0; j < MAX_TAPS - 1; ++j)
    if (j < n) tail[(int64_t)j * a.C + c] = v[j];
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
  float* red = qs + a.dk;            // [4][32]
  const int row = blockIdx.z, h = blockIdx.y, e0 = blockIdx.x * 32;
  const int tid = threadIdx.x, col = tid & 31, part = tid >> 5;
  const int e = e0 + col;
  const bool live = e < a.dv;
  const int64_t s0 = a.rows.start[row];
  const int len = (int)(a.rows.start[row + 1] - s0);
  float* Sg = a.S + ((int64_t)a.rows.slot[row] * a.H + h) * a.dk * a.dv;
  const bool first = row_pos0(a.rows, row) == 0;
  for (int i = part; i < a.dk; i += 4) S[i * 32 + col] = live && !first ? Sg[(int64_t)i * a.dv + e] : 0.f;
  const int kh = h / (a.H / a.KH);
  for (int t = 0; t < len; ++t) {
    const int64_t m = s0 + t;
    const float* cv = a.cv + m * a.ldc;
    __syncthreads();
    for (int i = tid; i < a.dk; i += 128) {
      ks[i] = cv[a.k_off + kh * a.dk + i];
      qs[i] = cv[a.q_off + kh * a.dk + i];
    }
    const float v = live ? cv[a.v_off + h * a.dv + e] : 0.f;
    const float g = expf(a.gl[m * a.H + h]), co = a.co[m * a.H + h];
    __syncthreads();
    float u = co * v;
    if (a.delta) {
      float p = 0.f;
      for (int i = part; i < a.dk; i += 4) {
        const float x = g * S[i * 32 + col];
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
      const float x = (a.delta ? S[i * 32 + col] : g * S[i * 32 + col]) + ks[i] * u;
      S[i * 32 + col] = x;
      o += x * qs[i];
    }
    red[part * 32 + col] = o;
    __syncthreads();
    if (part == 0 && live) {
      o = (red[col] + red[32 + col]) + (red[64 + col] + red[96 + col]);
      if (a.dskip) o += a.dskip[h] * v;
      a.o[m * (int64_t)a.H * a.dv + h * a.dv + e] = o;
    }
  }
  if (live)
    for (int i = part; i < a.dk; i += 4) Sg[(int64_t)i * a.dv + e] = S[i * 32 + col];
}

// delta: per head, rms over dv, plain weight, times silu(gate).  ssd: times silu(gate) first, then
// rms over each of norm_groups equal parts.  One block per (norm group, token).
template <class T>
__global__ void k_gated_norm(RecurArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __shared__ float sh[32];
  const int64_t m = blockIdx.y;
  const int n = a.delta ? a.dv : a.H * a.dv / a.norm_groups;
  const int c0 = blockIdx.x * n;
  const float* o = a.o + m * (int64_t)a.H * a.dv + c0;
  const float* gate = a.proj + m * a.ldp + a.gate_off + c0;
  T* out = (T*)a.att + m * a.ld_att + c0;
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float v = a.delta ? o[i] : o[i] * silu(gate[i]);
    ss += v * v;
  }
  ss = block_sum(ss, sh);
  const float rms = sqrtf(ss / (float)n + a.eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float g = silu(gate[i]);
    const float v = a.delta ? o[i] / rms * a.norm[i] * g : o[i] * g / rms * a.norm[c0 + i];
    st(out + i, v);
  }
}

}  // namespace

int k_launch_conv_heads(cg_ctx* c, const RecurArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  CG_CUDA(c, launch_kernel(c, k_conv_heads, dim3((unsigned)a.rows.M), dim3(256), 0, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_conv_tail(cg_ctx* c, const RecurArgs& a) {
  if (a.rows.M == 0 || a.taps <= 1) return CG_OK;
  if (a.taps > MAX_TAPS) return fail(c, CG_ERR_UNSUPPORTED, "recurrence: too many convolution taps");
  CG_CUDA(c, launch_kernel(c, k_conv_tail, dim3((unsigned)((a.C + 127) / 128), (unsigned)a.rows.rows), dim3(128), 0, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_recur_steps(cg_ctx* c, const RecurArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  const size_t smem = (size_t)(a.dk * 34 + 128) * 4;
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

int k_launch_gated_norm(cg_ctx* c, const RecurArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  const int parts = a.delta ? a.H : a.norm_groups;
  const int n = a.H * a.dv / parts;
  const int block = std::min(512, (n + 31) / 32 * 32);
  dim3 grid((unsigned)parts, (unsigned)a.rows.M);
  if (grid.y > 65535) return fail(c, CG_ERR_UNSUPPORTED, "recurrence: too many tokens in one portion");
  if (a.bf16) CG_CUDA(c, launch_kernel(c, k_gated_norm<__nv_bfloat16>, grid, dim3(block), 0, 1, a));
  else CG_CUDA(c, launch_kernel(c, k_gated_norm<float>, grid, dim3(block), 0, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace cg
