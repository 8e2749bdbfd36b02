// chunk_common.cuh — what the kernels that run matrix-state recurrences in chunks of 64 tokens share: operand
// fragments, splits of f32 operands into two bf16 parts, and the inverse of a unit lower triangular matrix.
#pragma once

#include "mma.cuh"

namespace cg {

constexpr int CT = 64;   // tokens per chunk
constexpr int EB = 64;   // value columns per block
constexpr int LE = EB + 8, LT = CT + 8;

__device__ __forceinline__ uint32_t sm_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

// v = hi + lo, both bf16
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *(const uint32_t*)&h;
  lo = *(const uint32_t*)&l;
}

// A fragment (16 x 16) of a row-major tile at (r0, c0)
__device__ __forceinline__ void frag_a(uint32_t base, int ld, int r0, int c0, int lane, uint32_t* a) {
  const int r = r0 + (lane & 7) + 8 * ((lane >> 3) & 1), c = c0 + 8 * (lane >> 4);
  ldsm_x4(base + (uint32_t)(r * ld + c) * 2u, a[0], a[1], a[2], a[3]);
}
// A fragment of the transpose: the tile is stored [k][m], fragment rows m0.., columns k0..
__device__ __forceinline__ void frag_a_t(uint32_t base, int ld, int m0, int k0, int lane, uint32_t* a) {
  const int k = k0 + (lane & 7) + 8 * (lane >> 4), m = m0 + 8 * ((lane >> 3) & 1);
  ldsm_x4_t(base + (uint32_t)(k * ld + m) * 2u, a[0], a[1], a[2], a[3]);
}
// B fragments of two neighbouring 8-column tiles; the operand is stored [k][n] ...
__device__ __forceinline__ void frag_b_kn(uint32_t base, int ld, int k0, int n0, int lane, uint32_t* b) {
  const int k = k0 + (lane & 7) + 8 * ((lane >> 3) & 1), n = n0 + 8 * (lane >> 4);
  ldsm_x4_t(base + (uint32_t)(k * ld + n) * 2u, b[0], b[1], b[2], b[3]);
}
// ... or [n][k]
__device__ __forceinline__ void frag_b_nk(uint32_t base, int ld, int k0, int n0, int lane, uint32_t* b) {
  const int n = n0 + (lane & 7) + 8 * (lane >> 4), k = k0 + 8 * ((lane >> 3) & 1);
  ldsm_x4(base + (uint32_t)(n * ld + k) * 2u, b[0], b[1], b[2], b[3]);
}

// 2^x to about 22 bits; its arguments here are at most 0
__device__ __forceinline__ float pow2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}


// X = (I + A)^-1 of the strictly lower triangular A, both [64][CHUNK_LD] f32 in shared memory, by `threads` >= 128
// threads of the block; A's upper half is scratch.  Begins and ends with the block in step.
constexpr int CHUNK_LD = 68;
__device__ __forceinline__ void invert_unit_lower(float* A, float* X, int tid, int threads) {
  // inverse by doubling blocks: four 16 x 16 diagonal blocks by substitution (one column per thread),
  // then [T1 0; -T2 A21 T1, T2] for 32 and for 64
  for (int i = tid; i < CT * CT; i += threads) X[(i >> 6) * CHUNK_LD + (i & 63)] = 0.f;
  __syncthreads();
  if (tid < CT) {
    const int b0 = tid & ~15, jc = tid & 15;
    float x[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float v = i == jc ? 1.f : 0.f;
#pragma unroll
      for (int s = 0; s < i; ++s) v -= A[(b0 + i) * CHUNK_LD + b0 + s] * x[s];  // x[s] = 0 above the diagonal
      x[i] = v;
      X[(b0 + i) * CHUNK_LD + tid] = v;
    }
  }
  __syncthreads();
  // Y[n x n] = L[n x n] Rm[n x n] (n 16 or 32): a thread takes one row and NC columns
  auto product = [&](const float* Lm, int ldl, const float* Rm, int ldr, float* Y, int ldy, int n, float sign, int u) {
    const int per_row = n / 8, r = u / per_row, c = (u - r * per_row) * 8;
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
#pragma unroll 4
    for (int k = 0; k < n; ++k) {
      const float l = Lm[r * ldl + k];
      const float4 r0 = *(const float4*)(Rm + k * ldr + c), r1 = *(const float4*)(Rm + k * ldr + c + 4);
      acc[0] += l * r0.x; acc[1] += l * r0.y; acc[2] += l * r0.z; acc[3] += l * r0.w;
      acc[4] += l * r1.x; acc[5] += l * r1.y; acc[6] += l * r1.z; acc[7] += l * r1.w;
    }
    *(float4*)(Y + r * ldy + c) = make_float4(sign * acc[0], sign * acc[1], sign * acc[2], sign * acc[3]);
    *(float4*)(Y + r * ldy + c + 4) = make_float4(sign * acc[4], sign * acc[5], sign * acc[6], sign * acc[7]);
  };
  {
    // two pairs of 16-blocks, 32 threads each; the products pass through the free upper blocks of A
    const int pr = tid >> 5, u = tid & 31, b = pr * 32;
    if (pr < 2) product(A + (b + 16) * CHUNK_LD + b, CHUNK_LD, X + b * CHUNK_LD + b, CHUNK_LD, A + b * CHUNK_LD + b + 16, CHUNK_LD, 16, 1.f, u);
    __syncthreads();
    if (pr < 2) product(X + (b + 16) * CHUNK_LD + b + 16, CHUNK_LD, A + b * CHUNK_LD + b + 16, CHUNK_LD, X + (b + 16) * CHUNK_LD + b, CHUNK_LD, 16, -1.f, u);
    __syncthreads();
    if (tid < 128) product(A + 32 * CHUNK_LD, CHUNK_LD, X, CHUNK_LD, A + 32, CHUNK_LD, 32, 1.f, tid);
    __syncthreads();
    if (tid < 128) product(X + 32 * CHUNK_LD + 32, CHUNK_LD, A + 32, CHUNK_LD, X + 32 * CHUNK_LD, CHUNK_LD, 32, -1.f, tid);
  }
  __syncthreads();
}

}  // namespace cg
