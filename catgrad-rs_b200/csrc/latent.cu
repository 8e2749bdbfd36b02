// latent.cu — attention whose keys and values are linear maps of one cached low-rank row per token
// (plus a rotated key part shared by all heads).
#include <algorithm>

#include "mixers.h"

namespace cg {

namespace {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
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
__device__ __forceinline__ float block_max(float v, float* sh) {
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = blockDim.x >> 5;
  v = warp_max(v);
  __syncthreads();
  if (lane == 0) sh[wid] = v;
  __syncthreads();
  v = lane < nw ? sh[lane] : -INFINITY;
  return warp_max(v);
}
__device__ __forceinline__ float ld(const float* p) { return *p; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void st4(float* p, float4 v) { *(float4*)p = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *(uint2*)p = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
}

// One block per token: the latent is normed and appended with the rotated key part; the queries'
// rotated parts are rotated and laid out head by head with Dq values each.
template <class T>
__global__ void __launch_bounds__(256) k_latent_prep(LatentArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __shared__ float sh[32];
  const int64_t m = blockIdx.x;
  const int row = a.rows.tok_row[m];
  const int64_t pos = row_pos0(a.rows, row) + (m - a.rows.start[row]);
  const float* p = a.proj + m * a.ldp;
  const float* dk = p + a.dkv_off;
  T* crow = (T*)a.cache + ((int64_t)a.rows.slot[row] * a.Tmax + pos) * a.Lw;
  T* cpk = a.c_out ? (T*)a.c_out + m * a.Lw : nullptr;
  const int half = a.r / 2;
  const float* ct = a.cos_t + pos * half;
  const float* sn = a.sin_t + pos * half;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.R; i += blockDim.x) ss += dk[i] * dk[i];
  ss = block_sum(ss, sh);
  const float rms = sqrtf(ss / (float)a.R + a.eps);
  for (int i = threadIdx.x; i < (int)a.Lw; i += blockDim.x) {
    float v = 0.f;
    if (i < a.R) v = dk[i] / rms * a.c_gain[i];
    else if (i < a.R + a.r) {
      const int j = i - a.R, k = j >> 1;
      const float u = dk[a.R + 2 * k], w = dk[a.R + 2 * k + 1];
      v = (j & 1) ? w * ct[k] + u * sn[k] : u * ct[k] - w * sn[k];
    }
    st(crow + i, v);
    if (cpk) st(cpk + i, v);
  }
  const int D = a.d + a.r, total = a.H * a.Dq;
  T* q = (T*)a.q_out + m * (int64_t)total;
  if (((a.d | a.Dq | D) & 3) == 0 && (a.ldp & 3) == 0) {
    // four values at a time
    for (int i = 4 * threadIdx.x; i < total; i += 4 * blockDim.x) {
      const int h = i / a.Dq, e = i - h * a.Dq;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (e < D) v = *(const float4*)(p + h * D + e);
      if (e >= a.d && e < D) {
        const int k = (e - a.d) >> 1;
        const float2 c = *(const float2*)(ct + k), s = *(const float2*)(sn + k);
        v = make_float4(v.x * c.x - v.y * s.x, v.y * c.x + v.x * s.x, v.z * c.y - v.w * s.y, v.w * c.y + v.z * s.y);
      }
      st4(q + i, v);
    }
    return;
  }
  for (int i = threadIdx.x; i < total; i += blockDim.x) {
    const int h = i / a.Dq, e = i - h * a.Dq;
    const float* qh = p + h * D;
    float v = 0.f;
    if (e < a.d) v = qh[e];
    else if (e < D) {
      const int j = e - a.d, k = j >> 1;
      const float u = qh[a.d + 2 * k], w = qh[a.d + 2 * k + 1];
      v = (j & 1) ? w * ct[k] + u * sn[k] : u * ct[k] - w * sn[k];
    }
    st(q + i, v);
  }
}

// One block per (token, head), any sizes: the query is mapped through Wuk into the cached rows'
// space, an online softmax runs over tiles of cached rows, and the result is mapped through Wuv.
template <class T>
__global__ void __launch_bounds__(256) k_latent_attn(LatentArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  constexpr int KT = 64;
  extern __shared__ float sm[];
  const int64_t m = blockIdx.x;
  const int h = blockIdx.y;
  const int row = a.rows.tok_row[m];
  const int64_t pos = row_pos0(a.rows, row) + (m - a.rows.start[row]);
  const int Lr = a.R + a.r;
  float* q = sm;            // [d + r]
  float* qa = q + a.d + a.r;  // [R + r]
  float* o = qa + Lr;       // [R]
  float* s = o + a.R;       // [KT]
  float* sh = s + KT;       // [32]
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
  const T* qg = (const T*)a.q_out + m * (int64_t)a.H * a.Dq + (int64_t)h * a.Dq;
  for (int i = tid; i < a.d + a.r; i += blockDim.x) q[i] = ld(qg + i);
  __syncthreads();
  const T* uk = (const T*)a.uk + (int64_t)h * a.d * a.R;
  for (int i = tid; i < a.R; i += blockDim.x) {
    float v = 0.f;
    for (int e = 0; e < a.d; ++e) v += q[e] * ld(uk + (int64_t)e * a.R + i);
    qa[i] = v;
    o[i] = 0.f;
  }
  for (int i = tid; i < a.r; i += blockDim.x) qa[a.R + i] = q[a.d + i];
  __syncthreads();
  const T* base = (const T*)a.cache + (int64_t)a.rows.slot[row] * a.Tmax * a.Lw;
  float mx = -INFINITY, l = 0.f;
  for (int64_t k0 = 0; k0 <= pos; k0 += KT) {
    const int n = (int)min((int64_t)KT, pos + 1 - k0);
    for (int j = warp; j < n; j += nw) {
      const T* kr = base + (k0 + j) * a.Lw;
      float v = 0.f;
      for (int i = lane; i < Lr; i += 32) v += qa[i] * ld(kr + i);
      v = warp_sum(v);
      if (lane == 0) s[j] = v * a.scale;
    }
    __syncthreads();
    float t = -INFINITY;
    for (int j = tid; j < n; j += blockDim.x) t = fmaxf(t, s[j]);
    const float mn = fmaxf(mx, block_max(t, sh));
    const float corr = mx == -INFINITY ? 0.f : expf(mx - mn);
    float ls = 0.f;
    for (int j = tid; j < n; j += blockDim.x) {
      const float e = expf(s[j] - mn);
      s[j] = e;
      ls += e;
    }
    l = l * corr + block_sum(ls, sh);  // (its barriers also publish s)
    mx = mn;
    for (int i = tid; i < a.R; i += blockDim.x) {
      float v = o[i] * corr;
      for (int j = 0; j < n; ++j) v += s[j] * ld(base + (k0 + j) * a.Lw + i);
      o[i] = v;
    }
    __syncthreads();
  }
  const float inv = 1.f / l;
  const T* uv = (const T*)a.uv + (int64_t)h * a.dv * a.R;
  T* out = (T*)a.att + m * a.ld_att + (int64_t)h * a.Do;
  for (int e = warp; e < a.dv; e += nw) {
    float v = 0.f;
    for (int i = lane; i < a.R; i += 32) v += o[i] * ld(uv + (int64_t)e * a.R + i);
    v = warp_sum(v);
    if (lane == 0) st(out + e, v * inv);
  }
}

}  // namespace

int k_launch_latent_prep(cg_ctx* c, const LatentArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  if (a.bf16) CG_CUDA(c, launch_kernel(c, k_latent_prep<__nv_bfloat16>, dim3((unsigned)a.rows.M), dim3(256), 0, 1, a));
  else CG_CUDA(c, launch_kernel(c, k_latent_prep<float>, dim3((unsigned)a.rows.M), dim3(256), 0, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_latent_attn(cg_ctx* c, const LatentArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  const size_t smem = (size_t)(a.d + a.r + 2 * a.R + a.r + 64 + 32) * 4;
  if (smem > 48 * 1024) return fail(c, CG_ERR_UNSUPPORTED, "latent attention: cached rows too wide");
  dim3 grid((unsigned)a.rows.M, (unsigned)a.H);
  if (a.bf16) CG_CUDA(c, launch_kernel(c, k_latent_attn<__nv_bfloat16>, grid, dim3(256), smem, 1, a));
  else CG_CUDA(c, launch_kernel(c, k_latent_attn<float>, grid, dim3(256), smem, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace cg
