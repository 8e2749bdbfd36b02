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
// u kept within +-limit.  One projection: ACT_RELU2 is the square of relu.
enum Act : int { ACT_SILU = 0, ACT_GELU = 1, ACT_BOUNDED = 2, ACT_RELU2 = 3 };
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

// What a GEMM stores in bf16: output mode 1 the product itself, 4 the square of its relu, 5 its silu.
__device__ __forceinline__ float bf16_out(int mode, float v) { return mode == 4 ? relu2_f(v) : mode == 5 ? silu_fast(v) : v; }

}  // namespace cg
