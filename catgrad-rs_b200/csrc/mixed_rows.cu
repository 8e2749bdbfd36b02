// mixed_rows.cu — the residual stream of decoders built layer by layer: embedding, post-norm add,
// next pre-norm and the two-part rows of a looped input in one pass; the same for several streams
// joined by hyper-connections, which also takes the weighted sum over a token's experts; activations
// of the f32 form.
#include <algorithm>
#include <type_traits>

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
__device__ __forceinline__ void store4(float* p, const float* v) { *(float4*)p = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float* v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
  *(uint2*)p = make_uint2(*(const uint32_t*)&lo, *(const uint32_t*)&hi);
}


// v = v * inv * g + b for vector i of a row, b may be null
template <bool EXACT>
__device__ __forceinline__ void gain(float* v, float inv, const float* g, int i, int W, const float* b = nullptr) {
  if (EXACT) {
    const float4 w = *(const float4*)(g + 4 * i);
    v[0] *= inv * w.x; v[1] *= inv * w.y; v[2] *= inv * w.z; v[3] *= inv * w.w;
    if (b) {
      const float4 t = *(const float4*)(b + 4 * i);
      v[0] += t.x; v[1] += t.y; v[2] += t.z; v[3] += t.w;
    }
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = 4 * i + e < W ? v[e] * (inv * g[4 * i + e]) + (b ? b[4 * i + e] : 0.f) : 0.f;
  }
}

// The norm of a row whose vectors the block's threads hold: thread t has vectors t + j blockDim.x, the
// columns past W are zero and stay so.
template <int VEC, bool EXACT>
__device__ __forceinline__ void norm_row(float (*v)[4], int centred, float eps, const float* g, const float* b, int nv, int n4, int W,
                                         float* sh) {
  if (centred) {
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < VEC; ++j) s += (v[j][0] + v[j][1]) + (v[j][2] + v[j][3]);
    const float mean = block_sum(s, sh) / (float)W;
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (j < nv && i < n4 && (EXACT || 4 * i + e < W)) v[j][e] -= mean;
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < VEC; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) ss += v[j][e] * v[j][e];
  ss = block_sum(ss, sh);
  const float inv = 1.f / sqrtf(ss / (float)W + eps);
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (j < nv && i < n4) gain<EXACT>(v[j], inv, g, i, W, b);
  }
}

// One block per row; the row lives in registers (RU_VEC 128-bit vectors per thread).
// EXACT: W is a multiple of 8, so no column is padding and gains and table rows are read as vectors.
template <class T, int RU_VEC, bool EXACT>
__global__ void k_row_update(RowUpdate u, int32_t* err) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __shared__ float sh[32];
  const int64_t m = blockIdx.x;
  const int W = u.W, n4 = (W + 7) / 8 * 2;
  const int nv = (n4 + blockDim.x - 1) / blockDim.x;
  float v[RU_VEC][4];
  if (u.pick) {
    const float* row = u.x + (int64_t)u.pick[m] * u.ldx;
#pragma unroll
    for (int j = 0; j < RU_VEC; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      const float4 t = j < nv && i < n4 ? *(const float4*)(row + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
      v[j][0] = t.x; v[j][1] = t.y; v[j][2] = t.z; v[j][3] = t.w;
    }
  } else {
    uint32_t tok = 0;
    if (u.tokens) {
      tok = u.tokens[m];
      if (tok >= u.vocab) { if (threadIdx.x == 0) *err = DEV_INDEX; tok = 0; }
    }
    float4 old[RU_VEC];  // requested before the reduction
#pragma unroll
    for (int j = 0; j < RU_VEC; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      old[j] = u.add && j < nv && i < n4 ? *(const float4*)(u.x + m * u.ldx + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
      v[j][0] = v[j][1] = v[j][2] = v[j][3] = 0.f;
      if (j < nv && i < n4) {
        if (u.tokens) {
          const int64_t o = (int64_t)tok * W + 4 * i;
          if (EXACT && u.table_bf16) {
            const uint2 r = *(const uint2*)((const __nv_bfloat16*)u.table + o);
            const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&r.x), b = __bfloat1622float2(*(const __nv_bfloat162*)&r.y);
            v[j][0] = a.x; v[j][1] = a.y; v[j][2] = b.x; v[j][3] = b.y;
          } else
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (4 * i + e < W)
              v[j][e] = u.table_bf16 ? __bfloat162float(((const __nv_bfloat16*)u.table)[o + e]) : ((const float*)u.table)[o + e];
#pragma unroll
          for (int e = 0; e < 4; ++e) v[j][e] *= u.scale;
        } else {
          if (u.y) {
            const float4 t = *(const float4*)(u.y + m * u.ldy + 4 * i);
            v[j][0] = t.x; v[j][1] = t.y; v[j][2] = t.z; v[j][3] = t.w;
          }
          for (int q = 0; q < u.top; ++q) {
            const int r = u.pos[m * u.top + q];
            if (r < 0) continue;
            const float w = u.wts ? u.wts[m * u.top + q] : 1.f;
            const float4 t = *(const float4*)(u.ye + (int64_t)r * u.ldye + 4 * i);
            v[j][0] += w * t.x; v[j][1] += w * t.y; v[j][2] += w * t.z; v[j][3] += w * t.w;
          }
          if (!EXACT)
#pragma unroll
            for (int e = 0; e < 4; ++e)
              if (4 * i + e >= W) v[j][e] = 0.f;
        }
      }
    }
    if (u.g1) norm_row<RU_VEC, EXACT>(v, u.centred, u.eps, u.g1, u.b1, nv, n4, W, sh);
#pragma unroll
    for (int j = 0; j < RU_VEC; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (j < nv && i < n4) {
        float* xp = u.x + m * u.ldx + 4 * i;
        v[j][0] += old[j].x; v[j][1] += old[j].y; v[j][2] += old[j].z; v[j][3] += old[j].w;
        store4(xp, v[j]);
      }
    }
  }
  if (u.x0)
#pragma unroll
    for (int j = 0; j < RU_VEC; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (j < nv && i < n4) store4((T*)u.x0 + m * u.ld0 + 4 * i, v[j]);
    }
  if (!u.out) return;
  const int64_t mo = u.dst ? u.dst[m] : m;
  if (u.g2) norm_row<RU_VEC, EXACT>(v, u.centred, u.eps, u.g2, u.b2, nv, n4, W, sh);
#pragma unroll
  for (int j = 0; j < RU_VEC; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (j < nv && i < n4) store4((T*)u.out + mo * u.ldo + 4 * i, v[j]);
  }
}

// One block per token.  Vector i of all streams is read, mixed and written by one thread, which keeps
// its part of the next sublayer's input (VEC 128-bit vectors) for the norm.  NS bounds the streams.
template <class T, int NS, int VEC, bool EXACT>
__global__ void k_stream_update(StreamUpdate u, int32_t* err) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  __shared__ float sh[32];
  __shared__ float cf[NS * NS + 2 * NS];  // mix, out, in: weights, read before the wait
  const int64_t m = blockIdx.x;
  const int ns = u.ns, W = u.W, n4 = (W + 7) / 8 * 2;
  const int nv = (n4 + blockDim.x - 1) / blockDim.x;
  float *mix = cf, *ow = cf + NS * NS, *iw = ow + NS;
  for (int i = threadIdx.x; i < NS * NS + 2 * NS; i += blockDim.x) {
    float v = 0.f;
    if (i < NS * NS) {
      if (u.mix && i / NS < ns && i % NS < ns) v = u.mix[(i / NS) * ns + i % NS];
    } else if (i < NS * NS + NS) {
      if (u.out_w && i - NS * NS < ns) v = u.out_w[i - NS * NS];
    } else if (i - NS * NS - NS < ns) v = u.in_w ? u.in_w[i - NS * NS - NS] : 1.f;
    cf[i] = v;
  }
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __syncthreads();
  uint32_t tok = 0;
  if (u.tokens) {
    tok = u.tokens[m];
    if (tok >= u.vocab) { if (threadIdx.x == 0) *err = DEV_INDEX; tok = 0; }
  }
  float* const x0 = u.x + (u.pick ? (int64_t)u.pick[m] : m) * ns * u.ldx;
  float h[VEC][4];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    h[j][0] = h[j][1] = h[j][2] = h[j][3] = 0.f;
    if (j >= nv || i >= n4) continue;
    float x[NS][4], y[4] = {0.f, 0.f, 0.f, 0.f};
    if (u.tokens) {
      const int64_t o = (int64_t)tok * W + 4 * i;
      if (EXACT && u.table_bf16) {
        const uint2 r = *(const uint2*)((const __nv_bfloat16*)u.table + o);
        const float2 a = __bfloat1622float2(*(const __nv_bfloat162*)&r.x), b = __bfloat1622float2(*(const __nv_bfloat162*)&r.y);
        y[0] = a.x; y[1] = a.y; y[2] = b.x; y[3] = b.y;
      } else
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (4 * i + e < W)
            y[e] = u.table_bf16 ? __bfloat162float(((const __nv_bfloat16*)u.table)[o + e]) : ((const float*)u.table)[o + e];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        y[e] *= u.scale;
#pragma unroll
        for (int t = 0; t < NS; ++t) x[t][e] = y[e];
      }
    } else {
      float old[NS][4];
#pragma unroll
      for (int s = 0; s < NS; ++s) {
        const float4 v = s < ns ? *(const float4*)(x0 + s * u.ldx + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        old[s][0] = v.x; old[s][1] = v.y; old[s][2] = v.z; old[s][3] = v.w;
      }
      if (u.pick) {
#pragma unroll
        for (int t = 0; t < NS; ++t)
#pragma unroll
          for (int e = 0; e < 4; ++e) x[t][e] = old[t][e];
      } else {
        if (u.top) {
          for (int q = 0; q < u.top; ++q) {
            const int r = u.pos[m * u.top + q];
            if (r < 0) continue;
            const float w = u.wts[m * u.top + q];
            const float4 v = *(const float4*)(u.y + (int64_t)r * u.ldy + 4 * i);
            y[0] += w * v.x; y[1] += w * v.y; y[2] += w * v.z; y[3] += w * v.w;
          }
        } else {
          const float4 v = *(const float4*)(u.y + m * u.ldy + 4 * i);
          y[0] = v.x; y[1] = v.y; y[2] = v.z; y[3] = v.w;
        }
        if (!EXACT)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (4 * i + e >= W) y[e] = 0.f;
#pragma unroll
        for (int t = 0; t < NS; ++t)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            float v = ow[t] * y[e];
#pragma unroll
            for (int s = 0; s < NS; ++s) v += mix[s * NS + t] * old[s][e];
            x[t][e] = v;
          }
      }
    }
    float total[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int t = 0; t < NS; ++t) {
      if (t < ns && !u.pick) store4(x0 + t * u.ldx + 4 * i, x[t]);
      if (t < ns)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          h[j][e] += iw[t] * x[t][e];
          total[e] += x[t][e];
        }
    }
    if (u.sum)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (4 * i + e < W) u.sum[m * u.ld_sum + 4 * i + e] = total[e];
#pragma unroll
    for (int e = 0; e < 4; ++e) ss += h[j][e] * h[j][e];
  }
  if (!u.out) return;
  ss = block_sum(ss, sh);
  const float inv = 1.f / sqrtf(ss / (float)W + u.eps);
  T* const out = (T*)u.out + (u.dst ? (int64_t)u.dst[m] : m) * u.ldo;
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    const int i = threadIdx.x + j * blockDim.x;
    if (j < nv && i < n4) {
      gain<EXACT>(h[j], inv, u.g, i, W);
      store4(out + 4 * i, h[j]);
    }
  }
}

__global__ void k_affine(float* x, int64_t n, float f, float v) {
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) x[i] = x[i] * f + v;
}

__global__ void k_relu2_f32(float* x, int64_t n) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) x[i] = relu2_f(x[i]);
}

__global__ void k_glu_f32(const float* gu, int64_t F, int act, float* out) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int64_t m = blockIdx.y;
  const float c = 0.7978845608028654f;  // sqrt(2 / pi)
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < F; i += (int64_t)gridDim.x * blockDim.x) {
    const float z = gu[m * 2 * F + i];
    const float a = act == 0 ? z / (1.f + expf(-z)) : 0.5f * z * (1.f + tanhf(c * (z + 0.044715f * z * z * z)));
    out[m * F + i] = a * gu[m * 2 * F + F + i];
  }
}

__global__ void k_pair_rope_tables(PairRope f, int64_t T, int r, float* cos_t, float* sin_t) {
  const int half = r / 2;
  const int64_t n = T * half;
  for (int64_t i = blockIdx.x * (int64_t)blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t p = i / half;
    const int k = (int)(i - p * half);
    double w = pow(f.base, -2.0 * k / r);
    if (f.factor > 0) {
      const double turns = f.original * w / 6.283185307179586;  // of this pair over the original context
      if (turns < f.low) w /= f.factor;
      else if (turns <= f.high) {
        const double s = f.high > f.low ? (turns - f.low) / (f.high - f.low) : 1.0;
        w = (1.0 - s) * w / f.factor + s * w;
      }
    }
    const double a = (double)p * w;
    cos_t[i] = (float)cos(a);
    sin_t[i] = (float)sin(a);
  }
}

}  // namespace

int k_launch_row_update(cg_ctx* c, const RowUpdate& u, int64_t M, int out_bf16) {
  if (M == 0) return CG_OK;
  const int n4 = (u.W + 7) / 8 * 2;
  const bool exact = u.W % 8 == 0;
  const int vec = M <= 296 ? (n4 <= 1024 ? 1 : 4) : n4 <= 2048 ? 2 : 4;
  const int block = ((n4 + vec - 1) / vec + 31) / 32 * 32;
  if (block > 1024) return fail(c, CG_ERR_UNSUPPORTED, "decoder: rows wider than 16384 are not supported");
  auto pick = [&](auto t) {
    using T = decltype(t);
    if (exact) return vec == 1 ? k_row_update<T, 1, true> : vec == 2 ? k_row_update<T, 2, true> : k_row_update<T, 4, true>;
    return vec == 1 ? k_row_update<T, 1, false> : vec == 2 ? k_row_update<T, 2, false> : k_row_update<T, 4, false>;
  };
  auto kernel = out_bf16 ? pick(__nv_bfloat16()) : pick(float());
  CG_CUDA(c, launch_kernel(c, kernel, dim3((unsigned)M), dim3(block), 0, 1, u, c->core->dev_err));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_stream_update(cg_ctx* c, const StreamUpdate& u, int64_t M, int out_bf16) {
  if (M == 0) return CG_OK;
  const int n4 = (u.W + 7) / 8 * 2;
  const bool exact = u.W % 8 == 0;
  const int vec = M <= 296 ? (n4 <= 1024 ? 1 : 4) : n4 <= 2048 ? 2 : 4;
  const int block = ((n4 + vec - 1) / vec + 31) / 32 * 32;
  if (block > 1024) return fail(c, CG_ERR_UNSUPPORTED, "decoder: rows wider than 16384 are not supported");
  if (u.ns < 1 || u.ns > MAX_STREAMS) return fail(c, CG_ERR_UNSUPPORTED, "decoder: 1 to 16 streams");
  auto run = [&](auto t, auto ns) {
    using T = decltype(t);
    constexpr int NS = decltype(ns)::value;
    auto kernel = exact ? (vec == 1 ? k_stream_update<T, NS, 1, true> : vec == 2 ? k_stream_update<T, NS, 2, true> : k_stream_update<T, NS, 4, true>)
                        : (vec == 1 ? k_stream_update<T, NS, 1, false> : vec == 2 ? k_stream_update<T, NS, 2, false> : k_stream_update<T, NS, 4, false>);
    return launch_kernel(c, kernel, dim3((unsigned)M), dim3(block), 0, 1, u, c->core->dev_err);
  };
  auto pick = [&](auto t) {
    if (u.ns == 1) return run(t, std::integral_constant<int, 1>());
    if (u.ns == 2) return run(t, std::integral_constant<int, 2>());
    if (u.ns <= 4) return run(t, std::integral_constant<int, 4>());
    if (u.ns <= 8) return run(t, std::integral_constant<int, 8>());
    return run(t, std::integral_constant<int, 16>());
  };
  CG_CUDA(c, out_bf16 ? pick(__nv_bfloat16()) : pick(float()));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_affine(cg_ctx* c, float* x, int64_t n, float f, float v) {
  if (n == 0) return CG_OK;
  k_affine<<<grid_for(n, 256), 256, 0, c->core->stream>>>(x, n, f, v);
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_relu2_f32(cg_ctx* c, float* x, int64_t n) {
  if (n == 0) return CG_OK;
  CG_CUDA(c, launch_kernel(c, k_relu2_f32, dim3(grid_for(n, 256)), dim3(256), 0, 1, x, n));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_glu_f32(cg_ctx* c, const float* gu, int64_t M, int64_t F, int act, float* out) {
  if (M == 0) return CG_OK;
  CG_CUDA(c, launch_kernel(c, k_glu_f32, dim3(grid_for(F, 256, 64), (unsigned)M), dim3(256), 0, 1, gu, F, act, out));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_pair_rope_tables(cg_ctx* c, const PairRope& f, int64_t T, int r, float* cos_t, float* sin_t) {
  k_pair_rope_tables<<<grid_for(T * (r / 2), 256), 256, 0, c->core->stream>>>(f, T, r, cos_t, sin_t);
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace cg
