// rows_attn.cu — grouped-query attention on rows of unequal length: norms over all heads of the
// queries and of the keys or per head, rotation of neighbouring pairs and the cache append in one pass,
// and the attention of sizes (and of the f32 form) that the tensor-core kernels do not have.  Prompts in bf16
// take attention_fa.cu / attention.cu, decode steps attn_decode.cu.
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

// One block per token; Dk and Dv are multiples of 8, so four neighbours belong to one head.  A thread holds
// RQ vectors of the row at a time, all requested before the first is used.
// NORM: 0 none, 1 over all heads at once, 2 per head where one warp holds a head's vectors side by side,
// 3 per head of any size.
constexpr int RQ = 8, RQ_THREADS = 256;
template <class T, int NORM>
__global__ void __launch_bounds__(RQ_THREADS) k_rows_qkv(RowsAttnArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __shared__ float sh[32];
  extern __shared__ float per_head[];  // [H + G], NORM 3
  const int64_t m = blockIdx.x;
  const int row = a.rows.tok_row[m];
  const int64_t pos = row_pos0(a.rows, row) + (m - a.rows.start[row]);
  const int64_t slot = a.rows.slot[row];
  const float* p = a.proj + m * a.ldp;
  const int nq = a.H * a.Dk, nk = a.G * a.Dk, total = nq + nk + a.G * a.Dv;
  const int lanes = a.Dk / 4;
  float4 v[RQ];
  auto load = [&](int base) {
#pragma unroll
    for (int u = 0; u < RQ; ++u) {
      const int i = base + 4 * (threadIdx.x + u * RQ_THREADS);
      v[u] = i < total ? *(const float4*)(p + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load(0);
  float fq = 1.f, fk = 1.f;
  if (NORM == 1) {
    float sq = 0.f, sk = 0.f;
    auto add = [&](int i, float4 x) {
      const float s = x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
      if (i < nq) sq += s;
      else if (i < nq + nk) sk += s;
    };
#pragma unroll
    for (int u = 0; u < RQ; ++u) add(4 * (threadIdx.x + u * RQ_THREADS), v[u]);
    for (int i = 4 * (threadIdx.x + RQ * RQ_THREADS); i < nq + nk; i += 4 * RQ_THREADS) add(i, *(const float4*)(p + i));
    fq = 1.f / sqrtf(block_sum(sq, sh) / (float)(a.H * a.d) + a.eps);
    fk = 1.f / sqrtf(block_sum(sk, sh) / (float)(a.G * a.d) + a.eps);
  }
  if (NORM == 3) {
    const int lane = threadIdx.x & 31;
    for (int h = threadIdx.x >> 5; h < a.H + a.G; h += RQ_THREADS >> 5) {
      float ss = 0.f;
      for (int i = 4 * lane; i < a.Dk; i += 128) {
        const float4 x = *(const float4*)(p + h * a.Dk + i);
        ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
      }
      ss = warp_sum(ss);
      if (lane == 0) per_head[h] = 1.f / sqrtf(ss / (float)a.d + a.eps);
    }
    __syncthreads();
  }
  const int half = a.rot / 2;
  const float temp = a.q_temp ? a.q_temp[pos] : 1.f;
  const float* ct = a.cos_t + pos * half;
  const float* sn = a.sin_t + pos * half;
  T* const qo = (T*)a.q + m * nq;
  T* const ko = (T*)a.k_cache + (slot * a.G * a.Tmax + pos) * a.Dk;
  T* const vo = (T*)a.v_cache + (slot * a.G * a.Tmax + pos) * a.Dv;
  // head of a column: a shift where the head size is a power of two
  const int kshift = (a.Dk & (a.Dk - 1)) ? -1 : __ffs(a.Dk) - 1;
  for (int base = 0; base < total; base += 4 * RQ * RQ_THREADS) {
    if (base) load(base);
#pragma unroll
    for (int u = 0; u < RQ; ++u) {
      const int i = base + 4 * (threadIdx.x + u * RQ_THREADS);
      if (base + 4 * u * RQ_THREADS >= total) break;  // uniform over the block
      float4 x = v[u];
      if (NORM == 2) {
        float ss = x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
#pragma unroll
        for (int o = 16; o; o >>= 1) {
          const float t = __shfl_xor_sync(0xffffffffu, ss, o);
          if (o < lanes) ss += t;
        }
        if (i < nq + nk) {
          const float f = 1.f / sqrtf(ss / (float)a.d + a.eps);
          x = make_float4(x.x * f, x.y * f, x.z * f, x.w * f);
        }
      }
      if (i >= nq + nk) {
        if (i < total) {
          const int j = i - nq - nk, g = j / a.Dv;
          st4(vo + g * a.Tmax * a.Dv + (j - g * a.Dv), x);
        }
      } else {
        const bool is_q = i < nq;
        const int j = is_q ? i : i - nq, h = kshift >= 0 ? j >> kshift : j / a.Dk, e = j - h * a.Dk;
        if (NORM == 1) {
          const float f = is_q ? fq : fk;
          const float4 w = *(const float4*)((is_q ? a.q_gain : a.k_gain) + j);
          x = make_float4(x.x * (f * w.x), x.y * (f * w.y), x.z * (f * w.z), x.w * (f * w.w));
        } else if (NORM == 3) {
          const float f = per_head[is_q ? h : a.H + h];
          x = make_float4(x.x * f, x.y * f, x.z * f, x.w * f);
        }
        const int k = e >> 1;
        if (k < half) x = make_float4(x.x * ct[k] - x.y * sn[k], x.y * ct[k] + x.x * sn[k], x.z, x.w);
        if (k + 1 < half) x = make_float4(x.x, x.y, x.z * ct[k + 1] - x.w * sn[k + 1], x.w * ct[k + 1] + x.z * sn[k + 1]);
        if (is_q) {
          x = make_float4(x.x * temp, x.y * temp, x.z * temp, x.w * temp);
          st4(qo + i, x);
        }
        else st4(ko + h * a.Tmax * a.Dk + e, x);
      }
    }
  }
}

// One block per (token, head): an online softmax over tiles of the visible keys.
template <class T>
__global__ void __launch_bounds__(128) k_rows_attn(RowsAttnArgs a) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  constexpr int KT = 64;
  extern __shared__ float sm[];
  float* q = sm;          // [Dk]
  float* o = q + a.Dk;    // [Dv]
  float* s = o + a.Dv;    // [KT]
  float* sh = s + KT;     // [32]
  const int64_t m = blockIdx.x;
  const int h = blockIdx.y, g = h / (a.H / a.G);
  const int row = a.rows.tok_row[m];
  const int64_t pos = row_pos0(a.rows, row) + (m - a.rows.start[row]);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
  for (int i = tid; i < a.Dk; i += blockDim.x) q[i] = ld((const T*)a.q + (m * a.H + h) * a.Dk + i);
  for (int i = tid; i < a.Dv; i += blockDim.x) o[i] = 0.f;
  __syncthreads();
  const int64_t base = ((int64_t)a.rows.slot[row] * a.G + g) * a.Tmax;
  const T* kb = (const T*)a.k_cache + base * a.Dk;
  const T* vb = (const T*)a.v_cache + base * a.Dv;
  // the visible keys in sequence: the kf kept first ones, then [lo, pos]
  const int64_t lo = a.window > 0 ? max((int64_t)0, pos - a.window + 1) : 0, kf = min(a.keep_first, lo), end = kf + pos + 1 - lo;
  auto key = [&](int64_t v) { return v < kf ? v : v - kf + lo; };
  // the sink is a term of the sum before any key
  float mx = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.f : 0.f;
  for (int64_t k0 = 0; k0 < end; k0 += KT) {
    const int n = (int)min((int64_t)KT, end - k0);
    for (int j = warp; j < n; j += nw) {
      float v = 0.f;
      const T* kr = kb + key(k0 + j) * a.Dk;
      for (int i = lane; i < a.d; i += 32) v += q[i] * ld(kr + i);
      v = warp_sum(v);
      if (lane == 0) s[j] = v * a.scale - (a.bias ? a.bias[h * a.ld_bias + (pos - key(k0 + j))] : 0.f);
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
    for (int i = tid; i < a.dv; i += blockDim.x) {
      float v = o[i] * corr;
      for (int j = 0; j < n; ++j) v += s[j] * ld(vb + key(k0 + j) * a.Dv + i);
      o[i] = v;
    }
    __syncthreads();
  }
  T* out = (T*)a.att + m * a.ld_att + (int64_t)h * a.Dv;
  float f = a.out_scale;
  if (a.gate && !a.wide_gate) f *= 1.f / (1.f + expf(-a.gate[m * a.ldp + h]));
  for (int i = tid; i < a.Dv; i += blockDim.x)
    st(out + i, o[i] / l * (a.gate && a.wide_gate ? f / (1.f + expf(-a.gate[m * a.ldp + h * a.Dv + i])) : f));
}

}  // namespace

int k_launch_rows_qkv(cg_ctx* c, const RowsAttnArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  if (a.Dk % 8 || a.Dv % 8 || a.ldp % 4) return fail(c, CG_ERR_INVALID, "attention: head sizes must be padded to multiples of 8");
  const int lanes = a.Dk / 4;
  const int norm = a.q_gain ? 1 : !a.head_norm ? 0 : lanes == 2 || lanes == 4 || lanes == 8 || lanes == 16 || lanes == 32 ? 2 : 3;
  const size_t smem = norm == 3 ? (size_t)(a.H + a.G) * 4 : 0;
  if (smem > 40 * 1024) return fail(c, CG_ERR_UNSUPPORTED, "attention: too many heads");
  auto run = [&](auto t) {
    using T = decltype(t);
    auto kernel = norm == 0 ? k_rows_qkv<T, 0> : norm == 1 ? k_rows_qkv<T, 1> : norm == 2 ? k_rows_qkv<T, 2> : k_rows_qkv<T, 3>;
    return launch_kernel(c, kernel, dim3((unsigned)a.rows.M), dim3(RQ_THREADS), smem, 1, a);
  };
  CG_CUDA(c, a.bf16 ? run(__nv_bfloat16()) : run(float()));
  CG_LAUNCHED(c);
  return CG_OK;
}

int k_launch_rows_attn(cg_ctx* c, const RowsAttnArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  const size_t smem = (size_t)(a.Dk + a.Dv + 64 + 32) * 4;
  if (smem > 48 * 1024 || a.H > 65535) return fail(c, CG_ERR_UNSUPPORTED, "attention: heads too wide or too many");
  dim3 grid((unsigned)a.rows.M, (unsigned)a.H);
  if (a.bf16) CG_CUDA(c, launch_kernel(c, k_rows_attn<__nv_bfloat16>, grid, dim3(128), smem, 1, a));
  else CG_CUDA(c, launch_kernel(c, k_rows_attn<float>, grid, dim3(128), smem, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace cg
