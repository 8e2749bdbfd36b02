// channel_chunk.cu — prompts through the recurrences whose decay is a number per key channel (the delta rule
// and gated linear attention), 64 tokens at a time on the tensor cores.
//
// With G_t the running sum, per key channel, of the log decays inside a chunk (vectors of dk), S0 the state
// before it and u_t what token t writes,
//   S_t = diag(e^{G_t}) S0 + sum_{s<=t} diag(e^{G_t - G_s}) k_s u_s^T,        o_t = S_t^T q_t,
// and the pair products that couple tokens s <= t are  sum_c x_t[c] e^{G_t[c] - G_s[c]} k_s[c].  The exponential
// does not come out of the sum, and e^{-G_s} alone may overflow, so every pair gets a reference between
// its tokens: the chunk is halved three times, and for the pairs (upper half, lower half) of each
// halving the reference is the last token of the lower half: both factors are at most 1, whatever the
// decays.  What remains, pairs inside 8 tokens, is summed as it stands.
//
// For the delta rule (I + A) U = B (V - K~ S0) with K~ = e^G K, A_ts = b_t (pair product of k and k), B = diag(b).
// k_channel_prep makes T = (I + A)^-1 B, W = T K~ and U0 = T V for all chunks at once, so that the walk over
// chunks, k_channel_scan, has two dependent products per chunk:
//   U = U0 - W S0;   O = Q~ S0 + P U;   S = diag(e^{G_last}) S0 + K^^T U,   K^_s = e^{G_last - G_s} k_s
// (gated linear attention: U = V).
//
// Precision as in recurrent_chunk.cu: q, k, v are bf16; every f32 operand (state, P, T, W, U and the decayed
// q and k) is split into a bf16 head and remainder, accumulation is f32, the state is never rounded.
#include <algorithm>

#include "act.cuh"
#include "chunk_common.cuh"
#include "mixers.h"

namespace cg {

namespace {

// scratch of one (chunk, head), in bf16 values: [2][64][DK] of K^, Q~ and (delta) W, [2][64][64] of P
template <int DK, bool DELTA>
struct Scratch {
  static constexpr int64_t TILE = 2 * CT * DK;
  static constexpr int64_t KD = 0, QT = TILE, W = 2 * TILE, P = (DELTA ? 3 : 2) * TILE;
  static constexpr int64_t SIZE = P + 2 * CT * CT;
};

template <int DK>
struct PrepSmem {
  static constexpr int LK = DK + 8;
  static constexpr uint32_t K = 0;                               // [2][64][LK]
  static constexpr uint32_t KPART = CT * LK * 2;
  static constexpr uint32_t Q = 2 * KPART;                       // [2][32][LK] | X [64][68] f32
  static constexpr uint32_t QPART = 32 * LK * 2;
  static constexpr uint32_t QBYTES = 2 * QPART > CT * CHUNK_LD * 4 ? 2 * QPART : CT * CHUNK_LD * 4;
  static constexpr uint32_t A = Q + QBYTES;                      // [64][68] f32 | V [64][LE]
  static constexpr uint32_t P = A + CT * CHUNK_LD * 4;           // [64][68] f32 | T [2][64][LT]
  static constexpr uint32_t ENDS = P + 2 * CT * LT * 2;          // [8][DK] f32
  static constexpr uint32_t ROW = ENDS + 8 * DK * 4;             // beta, rq, rk [64] f32
  static constexpr uint32_t BYTES = ROW + 3 * CT * 4;
};

__device__ __forceinline__ float2 widen(uint32_t v) { return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u)); }

// v[0] of lane l becomes the sum over all lanes of value l / 2 of 16
__device__ __forceinline__ void reduce_scatter(float* v, int lane) {
#pragma unroll
  for (int n = 8; n; n >>= 1) {
    const bool upper = lane & (2 * n);
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i < n) {
        const float send = upper ? v[i] : v[i + n], keep = upper ? v[i + n] : v[i];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, 2 * n);
      }
  }
  v[0] += __shfl_xor_sync(0xffffffffu, v[0], 1);
}

// One block of 4 DK threads per (chunk, head).  A thread holds two neighbouring channels of 8 tokens: k and q
// as they are, and the running sums L of the log decays inside those tokens.
template <int DK, bool DELTA>
__global__ void __launch_bounds__(4 * DK, DK == 128 ? 2 : 4) k_channel_prep(ChunkArgs a) {
  using M = PrepSmem<DK>;
  using SC = Scratch<DK, DELTA>;
  constexpr int NT = 4 * DK, NW = NT / 32, LK = M::LK;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  extern __shared__ __align__(16) uint8_t smem[];
  const uint32_t base = sm_u32(smem);
  float* sA = (float*)(smem + M::A);
  float* sP = (float*)(smem + M::P);
  float* ends = (float*)(smem + M::ENDS);
  float *beta = (float*)(smem + M::ROW), *rq = beta + CT, *rk = rq + CT;
  const int chunk = blockIdx.x, h = blockIdx.y, kh = h / (a.H / a.KH);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int len = a.chunk_len[chunk];
  const int64_t m0 = a.chunk_tok[chunk];
  const int c = 2 * (tid % (DK / 2)), od = tid / (DK / 2), t0 = 8 * od;

  uint32_t k[8], q[8];
  float2 L[8];
  {
    const bool in_k = c < a.DKp, in_z = c < a.zs;
    const float coef = a.coef[h] * 1.4426950408889634f;
    float2 zb = make_float2(0.f, 0.f);
    if (in_z) zb = *(const float2*)(a.z_bias + h * a.zs + c);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const bool in = t0 + i < len;
      const int64_t m = m0 + (in ? t0 + i : 0);
      k[i] = in && in_k ? *(const uint32_t*)(a.k + m * a.ldq + (int64_t)kh * a.DKp + c) : 0;
      q[i] = in && in_k ? *(const uint32_t*)(a.q + m * a.ldq + (int64_t)kh * a.DKp + c) : 0;
      L[i] = in && in_z ? *(const float2*)(a.gl + m * (int64_t)a.H * a.zs + h * a.zs + c) : make_float2(0.f, 0.f);
    }
    float2 sum = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (t0 + i < len && in_z) {
        sum.x -= coef * softplus_f(a.z_sign * (L[i].x + zb.x));
        sum.y -= coef * softplus_f(a.z_sign * (L[i].y + zb.y));
      }
      L[i] = sum;
    }
    *(float2*)(ends + od * DK + c) = sum;
  }
  for (int t = tid; t < CT; t += NT) {
    const bool in = t < len;
    beta[t] = DELTA && in ? a.co[(m0 + t) * a.H + h] : 0.f;
    rq[t] = !in ? 0.f : DELTA ? a.rq[(m0 + t) * a.KH + kh] : a.q_scale;
    rk[t] = !in ? 0.f : DELTA ? a.rk[(m0 + t) * a.KH + kh] : 1.f;
  }
  for (int i = tid; i < CT * CHUNK_LD; i += NT) sA[i] = sP[i] = 0.f;
  __syncthreads();
  // the log decays of groups [from, to) of 8 tokens
  auto between = [&](int from, int to) {
    float2 v = make_float2(0.f, 0.f);
    for (int j = from; j < to; ++j) {
      const float2 e = *(const float2*)(ends + j * DK + c);
      v.x += e.x; v.y += e.y;
    }
    return v;
  };

  // pairs inside 8 tokens: rows T0 .. T1 - 1, of row t first t products of k and k, then t + 1 of q and k
  auto inside = [&](auto t0_, auto t1_) {
    constexpr int T0 = decltype(t0_)::value, T1 = decltype(t1_)::value;
    constexpr int N = T1 * T1 - T0 * T0;
    static_assert(N <= 16, "values of one reduction");
    float v[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) v[i] = 0.f;
#pragma unroll
    for (int t = T0; t < T1; ++t) {
      const float2 kt = widen(k[t]), qt = widen(q[t]);
      float* row = v + (t * t - T0 * T0);
#pragma unroll
      for (int s = 0; s <= t; ++s) {
        float2 ks = widen(k[s]);
        if (s < t) {
          ks.x *= pow2(L[t].x - L[s].x);
          ks.y *= pow2(L[t].y - L[s].y);
          if (DELTA) row[s] = kt.x * ks.x + kt.y * ks.y;
        }
        row[t + s] = qt.x * ks.x + qt.y * ks.y;
      }
    }
    reduce_scatter(v, lane);
    const int at = lane >> 1;
    if (at < N && !(lane & 1)) {
      int t = T0;
      while ((t + 1) * (t + 1) - T0 * T0 <= at) ++t;
      const int j = at - (t * t - T0 * T0), r = t0 + t;
      // (at most two warps hold channels of the same tokens: their sum does not depend on their order)
      if (j < t) atomicAdd(sA + r * CHUNK_LD + t0 + j, v[0]);
      else atomicAdd(sP + r * CHUNK_LD + t0 + j - t, v[0]);
    }
  };
  inside(std::integral_constant<int, 0>(), std::integral_constant<int, 4>());
  inside(std::integral_constant<int, 4>(), std::integral_constant<int, 5>());
  inside(std::integral_constant<int, 5>(), std::integral_constant<int, 6>());
  inside(std::integral_constant<int, 6>(), std::integral_constant<int, 7>());
  inside(std::integral_constant<int, 7>(), std::integral_constant<int, 8>());

  auto put = [&](uint32_t at, uint32_t part, uint32_t v, float fx, float fy) {
    const float2 f = widen(v);
    uint32_t hi, lo;
    split2(f.x * fx, f.y * fy, hi, lo);
    *(uint32_t*)(smem + at) = hi;
    *(uint32_t*)(smem + at + part) = lo;
  };
  // 16 x 16 products of rows of an f32-split operand with rows of K
  auto product = [&](uint32_t rows, uint32_t part, int ar, int br, float (*acc)[4]) {
#pragma unroll
    for (int j = 0; j < 2; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll 2
    for (int kk = 0; kk < DK; kk += 16) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      frag_a(base + rows, LK, ar, kk, lane, ah);
      frag_a(base + rows + part, LK, ar, kk, lane, al);
      frag_b_nk(base + M::K, LK, kk, br, lane, bh);
      frag_b_nk(base + M::K + M::KPART, LK, kk, br, lane, bl);
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        mma_bf16(acc[y], ah[0], ah[1], ah[2], ah[3], bh[2 * y], bh[2 * y + 1]);
        mma_bf16(acc[y], ah[0], ah[1], ah[2], ah[3], bl[2 * y], bl[2 * y + 1]);
        mma_bf16(acc[y], al[0], al[1], al[2], al[3], bh[2 * y], bh[2 * y + 1]);
      }
    }
  };
  // halvings: HALF tokens of an upper half against the HALF before them
  auto halving = [&](auto half_) {
    constexpr int HALF = decltype(half_)::value;
    __syncthreads();  // the buffers are read
    constexpr int GROUPS = HALF / 8;
    const bool upper = od & GROUPS;          // uniform over the warp
    const int half0 = od & ~(GROUPS - 1);    // first group of this half
    const float2 far = upper ? between(half0, od) : between(od + 1, half0 + GROUPS);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int t = t0 + i;
      const float2 e = upper ? make_float2(far.x + L[i].x, far.y + L[i].y) : make_float2(far.x + (L[7].x - L[i].x), far.y + (L[7].y - L[i].y));
      const float fx = pow2(e.x), fy = pow2(e.y);
      if (DELTA || !upper) put(M::K + (uint32_t)(t * LK + c) * 2u, M::KPART, k[i], fx, fy);
      if (upper) put(M::Q + (uint32_t)(((t / (2 * HALF)) * HALF + (t & (HALF - 1))) * LK + c) * 2u, M::QPART, q[i], fx, fy);
    }
    __syncthreads();
    constexpr int UNITS = HALF == 16 ? 2 : 4;  // 16 x 16 (HALF 8: 8 x 8 inside) per operand
    for (int u = warp; u < 2 * UNITS; u += NW) {
      const bool is_q = u < UNITS;
      if (!is_q && !DELTA) break;
      const int b = u % UNITS;
      const int ar = HALF == 32 ? 32 + 16 * (b >> 1) : HALF == 16 ? 32 * b + 16 : 16 * b;           // rows of K
      const int qr = HALF == 32 ? 16 * (b >> 1) : HALF == 16 ? 16 * b : 16 * (b >> 1);               // rows of Q
      const int br = HALF == 32 ? 16 * (b & 1) : HALF == 16 ? 32 * b : 16 * b;
      float acc[2][4];
      if (is_q) product(M::Q, M::QPART, qr, br, acc);
      else product(M::K, M::KPART, ar, br, acc);
      float* out = is_q ? sP : sA;
#pragma unroll
      for (int y = 0; y < (HALF == 8 ? 1 : 2); ++y)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int r = (lane >> 2) + 8 * (e >> 1), s = br + y * 8 + (lane & 3) * 2 + (e & 1);
          if (HALF != 8) out[(ar + r) * CHUNK_LD + s] = acc[y][e];
          else if (is_q ? (r >> 3) == (b & 1) : r >= 8) out[(16 * b + 8 + (r & 7)) * CHUNK_LD + s] = acc[y][e];
        }
    }
  };
  halving(std::integral_constant<int, 32>());
  halving(std::integral_constant<int, 16>());
  halving(std::integral_constant<int, 8>());

  __nv_bfloat16* out = a.T + ((int64_t)chunk * a.H + h) * SC::SIZE;
  auto store = [&](int64_t tile, int t, float x, float y) {
    uint32_t hi, lo;
    split2(x, y, hi, lo);
    *(uint32_t*)(out + tile + t * DK + c) = hi;
    *(uint32_t*)(out + tile + CT * DK + t * DK + c) = lo;
  };
  {
    // to the chunk's start and to its end
    const float2 before = between(0, od), behind = between(od + 1, 8);
    const float2 last = L[7];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int t = t0 + i;
      const float2 kf = widen(k[i]), qf = widen(q[i]);
      const float fx = pow2(before.x + L[i].x), fy = pow2(before.y + L[i].y);
      store(SC::QT, t, qf.x * (rq[t] * fx), qf.y * (rq[t] * fy));
      store(SC::KD, t, kf.x * (rk[t] * pow2(behind.x + (last.x - L[i].x))), kf.y * (rk[t] * pow2(behind.y + (last.y - L[i].y))));
      if (DELTA) L[i] = make_float2(rk[t] * fx, rk[t] * fy);  // from here on the factor of K~
    }
    if (od == 7) *(float2*)(a.decayed + ((int64_t)chunk * a.H + h) * DK + c) = make_float2(pow2(before.x + last.x), pow2(before.y + last.y));
  }
  __syncthreads();  // pair products are complete, K and Q read
  for (int i = tid; i < CT * CT / 2; i += NT) {
    const int t = i / (CT / 2), s = (i - t * (CT / 2)) * 2;
    if (DELTA) {
      const float f = beta[t] * rk[t];
      sA[t * CHUNK_LD + s] *= f * rk[s];
      sA[t * CHUNK_LD + s + 1] *= f * rk[s + 1];
    }
    uint32_t hi, lo;
    split2(sP[t * CHUNK_LD + s] * (rq[t] * rk[s]), sP[t * CHUNK_LD + s + 1] * (rq[t] * rk[s + 1]), hi, lo);
    *(uint32_t*)(out + SC::P + t * CT + s) = hi;
    *(uint32_t*)(out + SC::P + CT * CT + t * CT + s) = lo;
  }
  if (!DELTA) return;
#pragma unroll
  for (int i = 0; i < 8; ++i) put(M::K + (uint32_t)((t0 + i) * LK + c) * 2u, M::KPART, k[i], L[i].x, L[i].y);
  __syncthreads();
  float* X = (float*)(smem + M::Q);
  invert_unit_lower(sA, X, tid, NT);
  for (int i = tid; i < CT * CT / 2; i += NT) {
    const int t = i / (CT / 2), s = (i - t * (CT / 2)) * 2;
    uint32_t hi, lo;
    split2(X[t * CHUNK_LD + s] * beta[s], X[t * CHUNK_LD + s + 1] * beta[s + 1], hi, lo);
    *(uint32_t*)(smem + M::P + (uint32_t)(t * LT + s) * 2u) = hi;
    *(uint32_t*)(smem + M::P + (uint32_t)(CT * LT + t * LT + s) * 2u) = lo;
  }
  __syncthreads();
  // W = T K~ and U0 = T V: a warp takes 16 tokens and every WN-th group of 16 columns
  constexpr int WN = NW / 4;
  const int wm = warp & 3, wn = warp >> 2, cq = (lane & 3) * 2, r_in = lane >> 2;
  auto t_times = [&](uint32_t right, uint32_t part, int ld, int n0, bool split, float (*acc)[4]) {
#pragma unroll
    for (int j = 0; j < 2; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    for (int kk = 0; kk <= wm * 16; kk += 16) {
      uint32_t th[4], tl[4], fh[4], fl[4];
      frag_a(base + M::P, LT, wm * 16, kk, lane, th);
      frag_a(base + M::P + CT * LT * 2, LT, wm * 16, kk, lane, tl);
      frag_b_kn(base + right, ld, kk, n0, lane, fh);
      if (split) frag_b_kn(base + right + part, ld, kk, n0, lane, fl);
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        mma_bf16(acc[y], th[0], th[1], th[2], th[3], fh[2 * y], fh[2 * y + 1]);
        mma_bf16(acc[y], tl[0], tl[1], tl[2], tl[3], fh[2 * y], fh[2 * y + 1]);
        if (split) mma_bf16(acc[y], th[0], th[1], th[2], th[3], fl[2 * y], fl[2 * y + 1]);
      }
    }
  };
  for (int n0 = wn * 16; n0 < DK; n0 += WN * 16) {
    float acc[2][4];
    t_times(M::K, M::KPART, LK, n0, true, acc);
#pragma unroll
    for (int y = 0; y < 2; ++y)
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int64_t o = SC::W + (int64_t)(wm * 16 + r_in + 8 * x) * DK + n0 + y * 8 + cq;
        uint32_t hi, lo;
        split2(acc[y][2 * x], acc[y][2 * x + 1], hi, lo);
        *(uint32_t*)(out + o) = hi;
        *(uint32_t*)(out + o + CT * DK) = lo;
      }
  }
  for (int e0 = 0; e0 < a.dv; e0 += EB) {
    __syncthreads();  // (A, and the columns before, are read)
    for (int i = tid; i < CT * (EB / 8); i += NT) {
      const int r = i / (EB / 8), n = (i - r * (EB / 8)) * 8;
      const bool in = r < len && e0 + n < a.dvp;
      cp_async16(base + M::A + (uint32_t)(r * LE + n) * 2u, a.v + (m0 + (in ? r : 0)) * a.ldv + (int64_t)h * a.dvp + (in ? e0 + n : 0), in ? 16 : 0);
    }
    cp_async_wait_all();
    __syncthreads();
    for (int n0 = wn * 16; n0 < EB && e0 + n0 < a.dvs; n0 += WN * 16) {
      float acc[2][4];
      t_times(M::A, 0, LE, n0, false, acc);
#pragma unroll
      for (int y = 0; y < 2; ++y)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int t = wm * 16 + r_in + 8 * x, n = e0 + n0 + y * 8 + cq;
          if (t < len && n < a.dvs)
            *(float2*)(a.o + (m0 + t) * (int64_t)a.H * a.dvs + (int64_t)h * a.dvs + n) = make_float2(acc[y][2 * x], acc[y][2 * x + 1]);
        }
    }
  }
}

// ------------------------------------------------------------------------ the walk ----
// Regions are reused inside a chunk so that two blocks share an SM: K^ takes W's place, P and U that of Q~.
template <int DK>
struct WalkSmem {
  static constexpr int LK = DK + 8;
  static constexpr uint32_t KPART = CT * LK * 2, UPART = CT * LE * 2, PPART = CT * LT * 2, SPART = DK * LE * 2;
  static constexpr uint32_t W = 0;                               // [2][64][LK]: W, then K^
  static constexpr uint32_t Q = 2 * KPART;                       // [2][64][LK] Q~ | P [2][64][LT], U [2][64][LE]
  static constexpr uint32_t P = Q, U = Q + 2 * PPART;
  static constexpr uint32_t QBYTES = 2 * KPART > 2 * PPART + 2 * UPART ? 2 * KPART : 2 * PPART + 2 * UPART;
  static constexpr uint32_t S = Q + QBYTES;                      // [2][DK][LE]
  static constexpr uint32_t D = S + 2 * SPART;                   // [DK] f32: e^{G_last}
  static constexpr uint32_t BYTES = D + DK * 4;
};

template <int DK, bool DELTA>
__global__ void __launch_bounds__(256, 2) k_channel_scan(ChunkArgs a) {
  using M = WalkSmem<DK>;
  using SC = Scratch<DK, DELTA>;
  constexpr int LK = M::LK;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  extern __shared__ __align__(16) uint8_t smem[];
  const uint32_t base = sm_u32(smem);
  float* dec = (float*)(smem + M::D);
  const int e0 = blockIdx.x * EB, h = blockIdx.y, row = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int wm = warp & 3, wn = warp >> 2;            // this warp's 16 tokens and 32 columns
  const int r_in = lane >> 2, cq = (lane & 3) * 2;
  const int c0 = a.row_chunk[row], c1 = a.row_chunk[row + 1];
  const bool first = row_pos0(a.rows, row) == 0;

  auto tile = [&](int chunk, int64_t from, uint32_t to) {  // [2][64][DK] into rows of LK
    const __nv_bfloat16* src = a.T + ((int64_t)chunk * a.H + h) * SC::SIZE + from;
    for (int i = tid; i < 2 * CT * (DK / 8); i += 256) {
      const int r = i / (DK / 8), x = i - r * (DK / 8);
      cp_async16(base + to + (uint32_t)(r * LK + x * 8) * 2u, src + r * DK + x * 8, 16);
    }
  };
  auto load = [&](int chunk) {
    tile(chunk, SC::QT, M::Q);
    tile(chunk, DELTA ? SC::W : SC::KD, M::W);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load(c0);

  constexpr int SN = DK == 128 ? 8 : 4;               // 8-column tiles a warp holds of 16 rows of the state
  const int sr = DK == 128 ? warp * 16 : wm * 16, sc = DK == 128 ? 0 : wn * 32;
  float S[SN][4];
  float* Sg = a.S + ((int64_t)a.rows.slot[row] * a.H + h) * a.dk * a.dvs;
#pragma unroll
  for (int j = 0; j < SN; ++j)
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int r = sr + r_in + 8 * b, n = e0 + sc + j * 8 + cq;
      float2 v = make_float2(0.f, 0.f);
      if (!first && r < a.dk && n < a.dvs) v = *(const float2*)(Sg + (int64_t)r * a.dvs + n);
      S[j][2 * b] = v.x; S[j][2 * b + 1] = v.y;
    }
  auto publish_state = [&]() {
#pragma unroll
    for (int j = 0; j < SN; ++j)
#pragma unroll
      for (int b = 0; b < 2; ++b) {
        uint32_t hi, lo;
        split2(S[j][2 * b], S[j][2 * b + 1], hi, lo);
        const uint32_t o = (uint32_t)((sr + r_in + 8 * b) * LE + sc + j * 8 + cq) * 2u;
        *(uint32_t*)(smem + M::S + o) = hi;
        *(uint32_t*)(smem + M::S + M::SPART + o) = lo;
      }
  };
  publish_state();

  for (int c = c0; c < c1; ++c) {
    const int len = a.chunk_len[c];
    const int64_t m0 = a.chunk_tok[c];
    const int t0 = wm * 16 + r_in;                    // this thread's tokens: t0 and t0 + 8
    auto at = [&](int x, int j) { return a.o + (m0 + t0 + 8 * x) * (int64_t)a.H * a.dvs + (int64_t)h * a.dvs + e0 + wn * 32 + j * 8 + cq; };
    auto there = [&](int x, int j) { return t0 + 8 * x < len && e0 + wn * 32 + j * 8 + cq < a.dvs; };
    float2 u0[4][2];
    if (DELTA)
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int x = 0; x < 2; ++x) u0[j][x] = there(x, j) ? *(const float2*)at(x, j) : make_float2(0.f, 0.f);
    const float d = tid < DK ? a.decayed[((int64_t)c * a.H + h) * DK + tid] : 0.f;
    cp_async_wait_all();
    __syncthreads();  // tiles and state of this chunk are in place
    float qs[4][4], ws[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) qs[j][e] = ws[j][e] = 0.f;
#pragma unroll 2
    for (int kk = 0; kk < DK; kk += 16) {
      uint32_t qh[4], ql[4], wh[4], wl[4];
      frag_a(base + M::Q, LK, wm * 16, kk, lane, qh);
      frag_a(base + M::Q + M::KPART, LK, wm * 16, kk, lane, ql);
      if (DELTA) {
        frag_a(base + M::W, LK, wm * 16, kk, lane, wh);
        frag_a(base + M::W + M::KPART, LK, wm * 16, kk, lane, wl);
      }
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        uint32_t fh[4], fl[4];
        frag_b_kn(base + M::S, LE, kk, wn * 32 + j * 8, lane, fh);
        frag_b_kn(base + M::S + M::SPART, LE, kk, wn * 32 + j * 8, lane, fl);
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          mma_bf16(qs[j + y], qh[0], qh[1], qh[2], qh[3], fh[2 * y], fh[2 * y + 1]);
          mma_bf16(qs[j + y], qh[0], qh[1], qh[2], qh[3], fl[2 * y], fl[2 * y + 1]);
          mma_bf16(qs[j + y], ql[0], ql[1], ql[2], ql[3], fh[2 * y], fh[2 * y + 1]);
          if (DELTA) {
            mma_bf16(ws[j + y], wh[0], wh[1], wh[2], wh[3], fh[2 * y], fh[2 * y + 1]);
            mma_bf16(ws[j + y], wh[0], wh[1], wh[2], wh[3], fl[2 * y], fl[2 * y + 1]);
            mma_bf16(ws[j + y], wl[0], wl[1], wl[2], wl[3], fh[2 * y], fh[2 * y + 1]);
          }
        }
      }
    }
    __syncthreads();  // Q~, W and the old state are read
    if (tid < DK) dec[tid] = d;
    {
      const __nv_bfloat16* src = a.T + ((int64_t)c * a.H + h) * SC::SIZE + SC::P;
      for (int i = tid; i < 2 * CT * (CT / 8); i += 256) {
        const int r = i / (CT / 8), x = i - r * (CT / 8);
        cp_async16(base + M::P + (uint32_t)(r * LT + x * 8) * 2u, src + r * CT + x * 8, 16);
      }
      if (DELTA) {
        tile(c, SC::KD, M::W);
      } else {
        for (int i = tid; i < CT * (EB / 8); i += 256) {
          const int r = i / (EB / 8), n = (i - r * (EB / 8)) * 8;
          const bool in = r < len && e0 + n < a.dvp;
          cp_async16(base + M::U + (uint32_t)(r * LE + n) * 2u, a.v + (m0 + (in ? r : 0)) * a.ldv + (int64_t)h * a.dvp + (in ? e0 + n : 0), in ? 16 : 0);
        }
      }
    }
    if (DELTA)
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          uint32_t hi, lo;
          split2(u0[j][x].x - ws[j][2 * x], u0[j][x].y - ws[j][2 * x + 1], hi, lo);
          const uint32_t o = (uint32_t)((t0 + 8 * x) * LE + wn * 32 + j * 8 + cq) * 2u;
          *(uint32_t*)(smem + M::U + o) = hi;
          *(uint32_t*)(smem + M::U + M::UPART + o) = lo;
        }
    cp_async_wait_all();
    __syncthreads();
    // O = Q~ S0 + P U
    for (int kk = 0; kk <= wm * 16; kk += 16) {
      uint32_t ph[4], pl[4];
      frag_a(base + M::P, LT, wm * 16, kk, lane, ph);
      frag_a(base + M::P + M::PPART, LT, wm * 16, kk, lane, pl);
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        uint32_t fh[4], fl[4];
        frag_b_kn(base + M::U, LE, kk, wn * 32 + j * 8, lane, fh);
        if (DELTA) frag_b_kn(base + M::U + M::UPART, LE, kk, wn * 32 + j * 8, lane, fl);
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          mma_bf16(qs[j + y], ph[0], ph[1], ph[2], ph[3], fh[2 * y], fh[2 * y + 1]);
          mma_bf16(qs[j + y], pl[0], pl[1], pl[2], pl[3], fh[2 * y], fh[2 * y + 1]);
          if (DELTA) mma_bf16(qs[j + y], ph[0], ph[1], ph[2], ph[3], fl[2 * y], fl[2 * y + 1]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int x = 0; x < 2; ++x)
        if (there(x, j)) *(float2*)at(x, j) = make_float2(qs[j][2 * x], qs[j][2 * x + 1]);
    // S = diag(e^{G_last}) S0 + K^^T U
    {
      const float f0 = dec[sr + r_in], f1 = dec[sr + r_in + 8];
#pragma unroll
      for (int j = 0; j < SN; ++j) { S[j][0] *= f0; S[j][1] *= f0; S[j][2] *= f1; S[j][3] *= f1; }
#pragma unroll
      for (int kk = 0; kk < CT; kk += 16) {
        uint32_t kh4[4], kl4[4];
        frag_a_t(base + M::W, LK, sr, kk, lane, kh4);
        frag_a_t(base + M::W + M::KPART, LK, sr, kk, lane, kl4);
#pragma unroll
        for (int j = 0; j < SN; j += 2) {
          uint32_t fh[4], fl[4];
          frag_b_kn(base + M::U, LE, kk, sc + j * 8, lane, fh);
          if (DELTA) frag_b_kn(base + M::U + M::UPART, LE, kk, sc + j * 8, lane, fl);
#pragma unroll
          for (int y = 0; y < 2; ++y) {
            mma_bf16(S[j + y], kh4[0], kh4[1], kh4[2], kh4[3], fh[2 * y], fh[2 * y + 1]);
            mma_bf16(S[j + y], kl4[0], kl4[1], kl4[2], kl4[3], fh[2 * y], fh[2 * y + 1]);
            if (DELTA) mma_bf16(S[j + y], kh4[0], kh4[1], kh4[2], kh4[3], fl[2 * y], fl[2 * y + 1]);
          }
        }
      }
    }
    if (c + 1 < c1) {
      __syncthreads();  // the chunk's tiles are read
      load(c + 1);
      publish_state();
    }
  }
#pragma unroll
  for (int j = 0; j < SN; ++j)
#pragma unroll
    for (int b = 0; b < 2; ++b) {
      const int r = sr + r_in + 8 * b, n = e0 + sc + j * 8 + cq;
      if (r < a.dk && n < a.dvs) *(float2*)(Sg + (int64_t)r * a.dvs + n) = make_float2(S[j][2 * b], S[j][2 * b + 1]);
    }
}

template <int DK, bool DELTA>
int launch_channel(cg_ctx* c, const ChunkArgs& a) {
  constexpr size_t prep = PrepSmem<DK>::BYTES, walk = WalkSmem<DK>::BYTES;
  static_assert(prep <= 113 * 1024 && walk <= 113 * 1024, "two blocks per SM");
  static PerDeviceFlag configured_on;
  bool& configured = configured_on.at(c->core->device);
  if (!configured) {
    CG_CUDA(c, cudaFuncSetAttribute(k_channel_prep<DK, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prep));
    CG_CUDA(c, cudaFuncSetAttribute(k_channel_scan<DK, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)walk));
    configured = true;
  }
  CG_CUDA(c, launch_kernel(c, k_channel_prep<DK, DELTA>, dim3((unsigned)a.n_chunks, (unsigned)a.H), dim3(4 * DK), prep, 1, a));
  CG_LAUNCHED(c);
  dim3 grid((unsigned)((a.dv + EB - 1) / EB), (unsigned)a.H, (unsigned)a.rows.rows);
  CG_CUDA(c, launch_kernel(c, k_channel_scan<DK, DELTA>, grid, dim3(256), walk, 1, a));
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace

int64_t channel_scratch(int dk, int delta) {
  if (dk <= 64) return delta ? Scratch<64, true>::SIZE : Scratch<64, false>::SIZE;
  return delta ? Scratch<128, true>::SIZE : Scratch<128, false>::SIZE;
}

int k_launch_channel_chunks(cg_ctx* c, const ChunkArgs& a) {
  if (a.rows.M == 0) return CG_OK;
  if (a.dk <= 64) return a.delta ? launch_channel<64, true>(c, a) : launch_channel<64, false>(c, a);
  return a.delta ? launch_channel<128, true>(c, a) : launch_channel<128, false>(c, a);
}

}  // namespace cg
