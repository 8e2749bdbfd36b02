// depth_rows.cu — the residual stream of designs whose sublayers run side by side on one norm: the sum of
// a layer's branches, the input a layer takes for the token itself, and the weighted average over the
// results of all layers so far, with the next layer's norm.
#include <algorithm>

#include "act.cuh"
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
__device__ __forceinline__ void store4(float* p, float4 v) { *(float4*)p = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *(uint2*)p = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
}
__device__ __forceinline__ void fma4(float4& a, float w, float4 v) {
  a.x += w * v.x; a.y += w * v.y; a.z += w * v.z; a.w += w * v.w;
}
__device__ __forceinline__ float dot4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
// four gains (or biases) of vector i, zero past column W
__device__ __forceinline__ float4 vec4(const float* p, int i, int W) {
  if (4 * i + 3 < W && (W & 3) == 0) return *(const float4*)(p + 4 * i);
  float v[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) v[e] = 4 * i + e < W ? p[4 * i + e] : 0.f;
  return make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ float4 scaled(float4 v, float f, float4 g) {
  return make_float4(v.x * f * g.x, v.y * f * g.y, v.z * f * g.z, v.w * f * g.w);
}

// One block per token; thread t has vectors t + j blockDim.x of the row.  Columns past W are zero in every
// operand (GEMM outputs of zero-padded weights) and stay so.
template <class T, int VEC>
__global__ void k_branch_sum(BranchSum u) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __shared__ float sh[32];
  const int64_t m = blockIdx.x;
  const int n4 = (u.W + 7) / 8 * 2;
  float4 acc[VEC], a[VEC], b[VEC];
  float sa = 0.f, sb = 0.f;
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    acc[j] = a[j] = b[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= n4) continue;
    acc[j] = *(const float4*)(u.x + m * u.ldx + 4 * i);
    if (u.normed[0]) {
      a[j] = *(const float4*)(u.normed[0] + m * u.ldy + 4 * i);
      b[j] = *(const float4*)(u.normed[1] + m * u.ldy + 4 * i);
      sa += dot4(a[j]);
      sb += dot4(b[j]);
    }
    if (u.y) fma4(acc[j], 1.f, *(const float4*)(u.y + m * u.ldy + 4 * i));
    if (u.y_bias) fma4(acc[j], 1.f, vec4(u.y_bias, i, u.W));
    for (int q = 0; q < u.top; ++q) {
      const int r = u.pos[m * u.top + q];
      if (r >= 0) fma4(acc[j], u.wts[m * u.top + q], *(const float4*)(u.ye + (int64_t)r * u.ldy + 4 * i));
    }
  }
  if (u.normed[0]) {
    sa = block_sum(sa, sh);
    sb = block_sum(sb, sh);
  }
  const float fa = 1.f / sqrtf(sa / (float)u.W + u.eps), fb = 1.f / sqrtf(sb / (float)u.W + u.eps);
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i >= n4) continue;
    if (u.normed[0]) {
      fma4(acc[j], 1.f, scaled(a[j], fa, vec4(u.gain[0], i, u.W)));
      fma4(acc[j], 1.f, scaled(b[j], fb, vec4(u.gain[1], i, u.W)));
    }
    store4(u.x + m * u.ldx + 4 * i, acc[j]);
    if (u.copy) store4((T*)u.copy + m * u.ld_copy + 4 * i, acc[j]);
  }
}

template <class T, int VEC>
__global__ void k_depth_update(DepthUpdate u, int32_t* err) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  __shared__ float sh[32];
  extern __shared__ float wts[];  // [n + 1]
  const int64_t m = blockIdx.x;
  const int W = u.W, n4 = (W + 7) / 8 * 2;
  for (int j = threadIdx.x; j <= u.n && u.average; j += blockDim.x) wts[j] = u.average[j];  // (weights: before the wait)
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __syncthreads();
  uint32_t tok = 0;
  if (u.tokens) {
    tok = u.tokens[m];
    if (tok >= u.vocab) { if (threadIdx.x == 0) *err = DEV_INDEX; tok = 0; }
  }
  float* const row = u.x + m * u.ldx;
  float4 v[VEC], y[VEC];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    v[j] = y[j] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= n4) continue;
    if (u.tokens) {
      float e[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int64_t o = (int64_t)tok * W + 4 * i + q;
        e[q] = 4 * i + q >= W ? 0.f : u.scale * (u.table_bf16 ? __bfloat162float(((const __nv_bfloat16*)u.table)[o]) : ((const float*)u.table)[o]);
      }
      v[j] = make_float4(e[0], e[1], e[2], e[3]);
    } else {
      v[j] = *(const float4*)(row + 4 * i);
      if (u.y) {
        y[j] = *(const float4*)(u.y + m * u.ldy + 4 * i);
        ss += dot4(y[j]);
      }
    }
  }
  if (u.y && !u.tokens) {
    const float f = 1.f / sqrtf(block_sum(ss, sh) / (float)W + u.eps);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < n4) fma4(v[j], 1.f, scaled(y[j], f, vec4(u.y_gain, i, W)));
    }
  }
  ss = 0.f;
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i >= n4) continue;
    float* d = u.depth + m * u.ldx + 4 * i;
    if (u.depth) store4(d + (int64_t)u.n * u.depth_stride, v[j]);
    if (u.average) {
      // the oldest first, as the sum is written; requests of four in flight
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
      int k = 0;
      for (; k + 4 <= u.n; k += 4) {
        float4 t[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) t[q] = *(const float4*)(d + (int64_t)(k + q) * u.depth_stride);
#pragma unroll
        for (int q = 0; q < 4; ++q) fma4(s, wts[k + q], t[q]);
      }
      for (; k < u.n; ++k) fma4(s, wts[k], *(const float4*)(d + (int64_t)k * u.depth_stride));
      fma4(s, wts[u.n], v[j]);
      v[j] = s;
    }
    store4(row + 4 * i, v[j]);
    if (u.kept)
#pragma unroll
      for (int q = 0; q < 4; ++q)
        if (4 * i + q < W) u.kept[m * u.ld_kept + 4 * i + q] = q == 0 ? v[j].x : q == 1 ? v[j].y : q == 2 ? v[j].z : v[j].w;
    ss += dot4(v[j]);
  }
  if (!u.out) return;
  const float f = 1.f / sqrtf(block_sum(ss, sh) / (float)W + u.eps);
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (i < n4) store4((T*)u.out + m * u.ldo + 4 * i, scaled(v[j], f, vec4(u.g, i, W)));
  }
}

__device__ __forceinline__ float gelu_as(float x, const float*) { return gelu_exact(x); }
__device__ __forceinline__ float gelu_as(float x, const __nv_bfloat16*) { return gelu_fast(x); }
// out[m, j] = gelu(z[m, j]) * table[token, off + j], zero past n.  `per` threads per token, neighbouring columns per
// thread.
__device__ __forceinline__ void st2(float* p, float a, float b) { *(float2*)p = make_float2(a, b); }
__device__ __forceinline__ void st2(__nv_bfloat16* p, float a, float b) { *(__nv_bfloat162*)p = __floats2bfloat162_rn(a, b); }
template <class T>
__global__ void __launch_bounds__(256) k_token_gate(TokenGate a, int64_t M, int per, int32_t* err) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int sub = threadIdx.x / per, t = threadIdx.x - sub * per;
  const int64_t m = (int64_t)blockIdx.x * (blockDim.x / per) + sub;
  if (m >= M) return;
  uint32_t tok = a.tokens[m];
  if (tok >= a.vocab) {
    if (t == 0) *err = DEV_INDEX;
    tok = 0;
  }
  const T* e = (const T*)a.table + (int64_t)tok * a.ld_table + a.off;
  T* out = (T*)a.out + m * a.ldo;
#pragma unroll 4
  for (int j = 2 * t; j < a.ldo; j += 2 * per) {
    const float2 z = *(const float2*)(a.z + m * a.ldz + j);
    const float e0 = j < a.n ? (float)e[j] : 0.f, e1 = j + 1 < a.n ? (float)e[j + 1] : 0.f;
    st2(out + j, gelu_as(z.x, (const T*)nullptr) * e0, gelu_as(z.y, (const T*)nullptr) * e1);
  }
}

__global__ void k_bias_gelu(const float* x, int64_t ldx, const float* bias, int64_t M, int64_t N, float* out, int64_t ldo) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < M * N; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t m = i / N, n = i - m * N;
    out[m * ldo + n] = gelu_exact(x[m * ldx + n] + bias[n]);
  }
}

// vectors a thread holds, and threads
struct Shape { int vec, block; };
Shape row_shape(int W, int64_t M) {
  const int n4 = (W + 7) / 8 * 2;
  const int vec = M <= 296 ? (n4 <= 1024 ? 1 : 4) : n4 <= 1024 ? 2 : 4;
  return {vec, ((n4 + vec - 1) / vec + 31) / 32 * 32};
}

}  // namespace

int k_launch_branch_sum(cg_ctx* c, const BranchSum& u, int64_t M, int bf16) {
  if (M == 0) return CG_OK;
  const Shape s = row_shape(u.W, M);
  if (s.block > 1024) return fail(c, CG_ERR_UNSUPPORTED, "decoder: rows wider than 16384 are not supported");
  auto pick = [&](auto t) {
    using T = decltype(t);
    return s.vec == 1 ? k_branch_sum<T, 1> : s.vec == 2 ? k_branch_sum<T, 2> : k_branch_sum<T, 4>;
  };
  CG_CUDA(c, launch_kernel(c, bf16 ? pick(__nv_bfloat16()) : pick(float()), dim3((unsigned)M), dim3(s.block), 0, 1, u));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_depth_update(cg_ctx* c, const DepthUpdate& u, int64_t M, int bf16) {
  if (M == 0) return CG_OK;
  const Shape s = row_shape(u.W, M);
  if (s.block > 1024) return fail(c, CG_ERR_UNSUPPORTED, "decoder: rows wider than 16384 are not supported");
  const size_t smem = (size_t)(u.n + 1) * 4;
  if (smem > 40 * 1024) return fail(c, CG_ERR_UNSUPPORTED, "decoder: too many layers to average over");
  auto pick = [&](auto t) {
    using T = decltype(t);
    return s.vec == 1 ? k_depth_update<T, 1> : s.vec == 2 ? k_depth_update<T, 2> : k_depth_update<T, 4>;
  };
  CG_CUDA(c, launch_kernel(c, bf16 ? pick(__nv_bfloat16()) : pick(float()), dim3((unsigned)M), dim3(s.block), smem, 1, u, c->core->dev_err));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_token_gate(cg_ctx* c, const TokenGate& a, int64_t M, int bf16) {
  if (M == 0) return CG_OK;
  auto kernel = bf16 ? k_token_gate<__nv_bfloat16> : k_token_gate<float>;
  if (a.ldo % 2 || a.ldz % 2) return fail(c, CG_ERR_INVALID, "decoder: token inputs must be padded to pairs");
  const int per = M <= 296 ? 128 : 32, block = M <= 296 ? 128 : 256;
  CG_CUDA(c, launch_kernel(c, kernel, dim3((unsigned)((M + block / per - 1) / (block / per))), dim3(block), 0, 1, a, M, per, c->core->dev_err));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_bias_gelu_f32(cg_ctx* c, const float* x, int64_t ldx, const float* bias, int64_t M, int64_t N, float* out, int64_t ldo) {
  if (M == 0) return CG_OK;
  CG_CUDA(c, launch_kernel(c, k_bias_gelu, dim3(grid_for(M * N, 256)), dim3(256), 0, 1, x, ldx, bias, M, N, out, ldo));
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace cg
