// act.cuh — the activation functions spelled the way catgrad's stdlib composes them
// (catgrad/src/stdlib/nn/mod.rs:130-160): sigmoid = 1 / (1 + exp(-x)), tanh = 2 sigmoid(2x) - 1,
// silu = x sigmoid(x), gelu = 0.5 x (1 + tanh(sqrt(2/pi) (x + 0.044715 x^3))).
#pragma once

namespace cg {

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + __expf(-x)); }
__device__ __forceinline__ float tanh_f(float x) { return 2.f * sigmoid_f(2.f * x) - 1.f; }
__device__ __forceinline__ float silu_f(float x) { return x * sigmoid_f(x); }
__device__ __forceinline__ float gelu_f(float x) {
  const float c = 0.7978845608f;  // sqrt(2/pi) in f32
  return 0.5f * x * (1.f + tanh_f(c * (x + 0.044715f * x * x * x)));
}

// Cheaper forms for epilogues whose result is rounded to bf16 anyway: approximate division.
__device__ __forceinline__ float sigmoid_fast(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
__device__ __forceinline__ float silu_fast(float x) { return x * sigmoid_fast(x); }
__device__ __forceinline__ float gelu_fast(float x) {
  const float c = 0.7978845608f;
  return 0.5f * x * (2.f * sigmoid_fast(2.f * c * (x + 0.044715f * x * x * x)));
}

// What a feed-forward applies to its projections (cg_act, include/catgrad_cuda.h).  Two projections:
// ACT_SILU and ACT_GELU gate the second one, ACT_BOUNDED is min(g, limit) sigmoid(1.702 g) (u + 1) with
// u kept within +-limit.  One projection: ACT_RELU2 is the square of relu, ACT_GELU1 gelu.
enum Act : int { ACT_SILU = 0, ACT_GELU = 1, ACT_BOUNDED = 2, ACT_RELU2 = 3, ACT_GELU1 = 4 };
__device__ __forceinline__ float bounded_glu(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_f(1.702f * g) * (u + 1.f);
}
__device__ __forceinline__ float glu_f(int act, float limit, float g, float u) {
  return act == ACT_SILU ? silu_f(g) * u : act == ACT_GELU ? gelu_f(g) * u : bounded_glu(g, u, limit);
}
__device__ __forceinline__ float relu2_f(float x) {
  x = fmaxf(x, 0.f);
  return x * x;
}

// What a GEMM stores in bf16: output mode 1 the product itself, 4 the square of its relu, 5 its silu, 6 the
// gelu of its sum with bias[n].
__device__ __forceinline__ float bf16_out(int mode, float v, const float* bias, int64_t n) {
  return mode == 4 ? relu2_f(v) : mode == 5 ? silu_fast(v) : mode == 6 ? gelu_fast(v + bias[n]) : v;
}

// ln(1 + e^x) with a relative error of about 1e-6: with e = e^-|x| and s = e / (2 + e),
// ln(1 + e) = 2 artanh(s), whose power series in s <= 1 / 3 needs eight terms.
__device__ __forceinline__ float softplus_f(float x) {
  const float e = __expf(-fabsf(x)), s = __fdividef(e, 2.f + e), q = s * s;
  float p = 1.f / 15.f;
  p = fmaf(p, q, 1.f / 13.f);
  p = fmaf(p, q, 1.f / 11.f);
  p = fmaf(p, q, 1.f / 9.f);
  p = fmaf(p, q, 1.f / 7.f);
  p = fmaf(p, q, 1.f / 5.f);
  p = fmaf(p, q, 1.f / 3.f);
  p = fmaf(p, q, 1.f);
  return fmaxf(x, 0.f) + 2.f * s * p;
}
// tanh-gelu on accurate exponentials; (1 + tanh u) / 2 as a sigmoid keeps its digits where u is far below 0
__device__ __forceinline__ float gelu_exact(float x) {
  return x / (1.f + expf(-1.5957691216057308f * (x + 0.044715f * x * x * x)));
}

}  // namespace cg
