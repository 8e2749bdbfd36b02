// latent_decode.cu — latent attention for a few new tokens per row (a decode step) in a bf16 context.
//
// The scores q . (Wuk c) are taken as (Wuk^T q) . c, so all heads attend over the same cached rows
// [c, rotated key part] and the cache is read once per token instead of being expanded:
//
//   k_latent_absorb   one block per (head, 64 latent columns): Wuk^T q for every new token; the
//                     last blocks norm / rotate / append the tokens' own cached rows and rotate q
//   k_latent_dec      one block per (token, 16 heads, context slice): heads are the rows of the
//                     MMA tile; 64 cached rows at a time through two shared-memory buffers,
//                     online softmax.  The slices are a thread-block cluster and merge their partial
//                     outputs over distributed shared memory, each its share of the latent columns
//   k_latent_out      one block per (head, 16 values): Wuv on the merged output
#include <algorithm>

#include "mixers.h"
#include "mma.cuh"
#include "tc_common.cuh"

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

struct DecodeScratch {
  __nv_bfloat16* qa;   // [M, H, Lw] queries in the cached rows' space
  float* o;            // [M, H, R] attention output in the latent space
  int splits;
};

__global__ void __launch_bounds__(256) k_latent_absorb(LatentArgs a, DecodeScratch s, int col_blocks) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, M = (int)a.rows.M, D = a.d + a.r;
  const int nb = a.H * col_blocks;
  if ((int)blockIdx.x >= nb) {
    // the new tokens' cached rows and the rotated parts of their queries
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int64_t m = blockIdx.x - nb;
    const int row = a.rows.tok_row[m];
    const int64_t pos = row_pos0(a.rows, row) + (m - a.rows.start[row]);
    const float* p = a.proj + m * a.ldp;
    const float* dk = p + a.dkv_off;
    __nv_bfloat16* crow = (__nv_bfloat16*)a.cache + ((int64_t)a.rows.slot[row] * a.Tmax + pos) * a.Lw;
    const int half = a.r / 2;
    const float* ct = a.cos_t + pos * half;
    const float* sn = a.sin_t + pos * half;
    auto rotated = [&](const float* x, int j) {
      const int k = j >> 1;
      const float u = x[2 * k], w = x[2 * k + 1];
      return (j & 1) ? w * ct[k] + u * sn[k] : u * ct[k] - w * sn[k];
    };
    float ss = 0.f;
    for (int i = tid; i < a.R; i += 256) ss += dk[i] * dk[i];
    ss = block_sum(ss, sm);
    const float rms = sqrtf(ss / (float)a.R + a.eps);
    for (int i = tid; i < (int)a.Lw; i += 256) {
      const float v = i < a.R ? dk[i] / rms * a.c_gain[i] : i < a.R + a.r ? rotated(dk + a.R, i - a.R) : 0.f;
      crow[i] = __float2bfloat16_rn(v);
    }
    const int w = (int)a.Lw - a.R;
    for (int i = tid; i < a.H * w; i += 256) {
      const int h = i / w, j = i - h * w;
      s.qa[(m * a.H + h) * a.Lw + a.R + j] = __float2bfloat16_rn(j < a.r ? rotated(p + h * D + a.d, j) : 0.f);
    }
    return;
  }
  // Wuk^T q for 64 latent columns of one head, 8 tokens at a time: 64 columns x 4 slices of the head dimension
  const int h = blockIdx.x / col_blocks, c = (blockIdx.x % col_blocks) * 64 + (tid & 63), part = tid >> 6;
  float* red = sm;                                     // [8][4][64]
  float* q = red + 8 * 256;                            // [d][8]
  __nv_bfloat16* w = (__nv_bfloat16*)(q + 8 * a.d);    // [d][64]
  const __nv_bfloat16* uk = (const __nv_bfloat16*)a.uk + (int64_t)h * a.d * a.R;
#pragma unroll 8
  for (int e = part; e < a.d; e += 4) w[e * 64 + (tid & 63)] = c < a.R ? uk[(int64_t)e * a.R + c] : __float2bfloat16_rn(0.f);
  asm volatile("griddepcontrol.wait;" ::: "memory");   // (the weights do not depend on it)
  for (int m0 = 0; m0 < M; m0 += 8) {
    const int n = min(8, M - m0);
    for (int i = tid; i < 8 * a.d; i += 256) {
      const int k = i / a.d, e = i - k * a.d;
      q[e * 8 + k] = k < n ? a.proj[(int64_t)(m0 + k) * a.ldp + h * D + e] : 0.f;
    }
    __syncthreads();
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
    for (int e = part; e < a.d; e += 4) {
      const float x = __bfloat162float(w[e * 64 + (tid & 63)]);
      const float4 q0 = *(const float4*)(q + e * 8), q1 = *(const float4*)(q + e * 8 + 4);
      v[0] += q0.x * x; v[1] += q0.y * x; v[2] += q0.z * x; v[3] += q0.w * x;
      v[4] += q1.x * x; v[5] += q1.y * x; v[6] += q1.z * x; v[7] += q1.w * x;
    }
#pragma unroll
    for (int k = 0; k < 8; ++k) red[k * 256 + tid] = v[k];
    __syncthreads();
    for (int k = part; k < n; k += 4) {
      const float* r = red + k * 256 + (tid & 63);
      if (c < a.R) s.qa[((int64_t)(m0 + k) * a.H + h) * a.Lw + c] = __float2bfloat16_rn((r[0] + r[64]) + (r[128] + r[192]));
    }
    // (the next round's writes to red come after its first barrier)
  }
}

constexpr int MAX_SLICES = 8;  // a portable cluster
constexpr int LD_KT = 64;  // cached rows per tile

// NT: 8-column output tiles per warp (eight warps share the latent columns)
template <int NT>
__global__ void __launch_bounds__(256) k_latent_dec(LatentArgs a, DecodeScratch sc, int ldk) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  extern __shared__ __align__(16) uint8_t smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  {
    // Before the dependency wait: this slice's cached rows are asked into L2.  The position may be a
    // step old here and the newest row unwritten; a prefetch changes nothing but where bytes lie.
    const int row = a.rows.tok_row[blockIdx.x];
    int64_t n = row_pos0(a.rows, row);
    n = n < 0 ? 0 : n > a.Tmax ? a.Tmax : n;
    const int64_t per = ((n + sc.splits) / sc.splits + 15) / 16 * 16, lo = blockIdx.z * per;
    const int64_t hi = min(n, lo + min(per, (int64_t)2 * LD_KT));
    const char* p = (const char*)((const __nv_bfloat16*)a.cache + (int64_t)a.rows.slot[row] * a.Tmax * a.Lw);
    const int64_t b_hi = hi * a.Lw * 2;
    for (int64_t b = lo * a.Lw * 2 + tid * 128; b < b_hi; b += 256 * 128)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(p + b));
  }
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __nv_bfloat16* sq = (__nv_bfloat16*)smem;            // [16][ldk]
  __nv_bfloat16* sk = sq + 16 * ldk;                   // [2][64][ldk]
  __nv_bfloat16* sp = sk + 2 * LD_KT * ldk;            // [16][72]
  float* wm = (float*)(sp + 16 * 72);                  // [8][16] per-warp row maxima
  float* wl = wm + 128;                                // [8][16] per-warp row sums
  const int64_t m = blockIdx.x;
  const int h0 = blockIdx.y * 16, split = blockIdx.z;
  const int row = a.rows.tok_row[m];
  const int64_t pos = row_pos0(a.rows, row) + (m - a.rows.start[row]);
  const __nv_bfloat16* base = (const __nv_bfloat16*)a.cache + (int64_t)a.rows.slot[row] * a.Tmax * a.Lw;
  const int64_t n_keys = pos + 1;
  const int64_t per = ((n_keys + sc.splits - 1) / sc.splits + 15) / 16 * 16;
  const int64_t k_lo = split * per, k_hi = min(n_keys, k_lo + per);
  const int CH = (int)a.Lw / 8;
  const uint32_t sq_u = (uint32_t)__cvta_generic_to_shared(sq), sk_u = (uint32_t)__cvta_generic_to_shared(sk),
                 sp_u = (uint32_t)__cvta_generic_to_shared(sp);
  const int row_bytes = (int)a.Lw * 2;
  // a warp copies whole rows; rows past the slice are zeros
  auto load = [&](int64_t k0, int buf) {
    const char* src = (const char*)(base + k0 * a.Lw) + lane * 16;
    const int n = (int)min((int64_t)LD_KT, k_hi - k0);
    uint32_t dst = sk_u + (uint32_t)((buf * LD_KT + warp) * ldk) * 2u + lane * 16;
#pragma unroll
    for (int r = warp; r < LD_KT; r += 8, dst += (uint32_t)(8 * ldk) * 2u) {
      const char* p = src + (r < n ? r : 0) * row_bytes;
      const int bytes = r < n ? 16 : 0;
      for (int ch = lane; ch < CH; ch += 32) cp_async16(dst + (ch - lane) * 16, p + (ch - lane) * 16, bytes);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float o[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float mrow[2] = {-INFINITY, -INFINITY}, lrow[2] = {0.f, 0.f};
  const int r_in = lane >> 2, cq = (lane & 3) * 2;
  if (k_lo < k_hi) {
#pragma unroll
    for (int r = warp; r < 16; r += 8) {
      const bool in = h0 + r < a.H;
      const __nv_bfloat16* p = sc.qa + (m * a.H + (in ? h0 + r : 0)) * a.Lw;
      for (int ch = lane; ch < CH; ch += 32) cp_async16(sq_u + (uint32_t)(r * ldk + ch * 8) * 2u, p + ch * 8, in ? 16 : 0);
    }
    load(k_lo, 0);
    int buf = 0;
    for (int64_t k0 = k_lo; k0 < k_hi; k0 += LD_KT, buf ^= 1) {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
      __syncthreads();  // the tile is in place; the other buffer, sp, wm and wl are free
      if (k0 + LD_KT < k_hi) load(k0 + LD_KT, buf ^ 1);
      const uint32_t kb = sk_u + (uint32_t)(buf * LD_KT * ldk) * 2u;
      // scores of this warp's eight keys
      float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};  // two chains
#pragma unroll 4
      for (int kk = 0; kk < (int)a.Lw; kk += 32) {
        uint32_t q0, q1, q2, q3, p0 = 0, p1 = 0, p2 = 0, p3 = 0, b0, b1, b2, b3;
        const bool two = kk + 16 < (int)a.Lw;
        const int qr = (lane & 7) + 8 * ((lane >> 3) & 1), qc = 8 * (lane >> 4);
        ldsm_x4(sq_u + (uint32_t)(qr * ldk + kk + qc) * 2u, q0, q1, q2, q3);
        if (two) ldsm_x4(sq_u + (uint32_t)(qr * ldk + kk + 16 + qc) * 2u, p0, p1, p2, p3);
        // four 8-column groups of the warp's keys (the last two stay inside the padded row)
        const int kc = kk + 8 * (lane >> 3);
        ldsm_x4(kb + (uint32_t)((warp * 8 + (lane & 7)) * ldk + (two || lane < 16 ? kc : kk)) * 2u, b0, b1, b2, b3);
        mma_bf16(s, q0, q1, q2, q3, b0, b1);
        if (two) mma_bf16(s2, p0, p1, p2, p3, b2, b3);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) s[e] += s2[e];
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[e] = k0 + warp * 8 + cq + (e & 1) < k_hi ? s[e] * a.scale : -INFINITY;
        mx[e >> 1] = fmaxf(mx[e >> 1], s[e]);
      }
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        mx[x] = fmaxf(mx[x], __shfl_xor_sync(0xffffffffu, mx[x], 1));
        mx[x] = fmaxf(mx[x], __shfl_xor_sync(0xffffffffu, mx[x], 2));
        if ((lane & 3) == 0) wm[warp * 16 + r_in + 8 * x] = mx[x];
      }
      __syncthreads();
      float corr[2], ls[2] = {0.f, 0.f};
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        float t = mrow[x];
#pragma unroll
        for (int w = 0; w < 8; ++w) t = fmaxf(t, wm[w * 16 + r_in + 8 * x]);  // finite: the tile has a key
        corr[x] = expf(mrow[x] - t);
        mrow[x] = t;
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[e] = expf(s[e] - mrow[e >> 1]);
        ls[e >> 1] += s[e];
      }
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        ls[x] += __shfl_xor_sync(0xffffffffu, ls[x], 1);
        ls[x] += __shfl_xor_sync(0xffffffffu, ls[x], 2);
        if ((lane & 3) == 0) wl[warp * 16 + r_in + 8 * x] = ls[x];
        *(uint32_t*)(sp + (r_in + 8 * x) * 72 + warp * 8 + cq) = pack_bf16(s[2 * x], s[2 * x + 1]);
      }
      __syncthreads();
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        float t = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) t += wl[w * 16 + r_in + 8 * x];
        lrow[x] = lrow[x] * corr[x] + t;
      }
#pragma unroll
      for (int j = 0; j < NT; ++j) { o[j][0] *= corr[0]; o[j][1] *= corr[0]; o[j][2] *= corr[1]; o[j][3] *= corr[1]; }
#pragma unroll
      for (int kk = 0; kk < LD_KT; kk += 16) {
        uint32_t p0, p1, p2, p3;
        ldsm_x4(sp_u + (uint32_t)(((lane & 7) + 8 * ((lane >> 3) & 1)) * 72 + kk + 8 * (lane >> 4)) * 2u, p0, p1, p2, p3);
#pragma unroll
        for (int j = 0; j < NT; j += 2) {
          uint32_t b0, b1, b2, b3;
          const int key = kk + (lane & 7) + 8 * ((lane >> 3) & 1), col = (warp * NT + j) * 8 + 8 * (lane >> 4);
          ldsm_x4_t(kb + (uint32_t)(key * ldk + col) * 2u, b0, b1, b2, b3);
          mma_bf16(o[j], p0, p1, p2, p3, b0, b1);
          mma_bf16(o[j + 1], p0, p1, p2, p3, b2, b3);
        }
      }
    }
  }
  // partial outputs and {maximum, sum} per head, over the tiles (each CTA's own are read)
  const int ldo = NT * 64 + 4;                         // (columns past R are not read)
  float* so = (float*)sk;                              // [16][ldo]
  float2* sml = (float2*)wm;                           // [16]
  __syncthreads();
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    if (warp == 0 && (lane & 3) == 0) sml[r_in + 8 * x] = make_float2(mrow[x], lrow[x]);
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int col = (warp * NT + j) * 8 + cq;
#pragma unroll
      for (int y = 0; y < 2; ++y)
        if (col + y < ldo) so[(r_in + 8 * x) * ldo + col + y] = o[j][2 * x + y];
    }
  }
  const int ns = sc.splits;
  if (ns > 1) tc::cluster_sync_all();
  else __syncthreads();
  float* wt = (float*)(sml + 16);                      // [ns][16] weight of each slice
  if (tid < 16) {
    float2 v[MAX_SLICES];
    float mx = -INFINITY, l = 0.f;
    const uint32_t at = tc::smem_u32(sml + tid);
#pragma unroll
    for (int k = 0; k < MAX_SLICES; ++k) {
      v[k] = make_float2(-INFINITY, 0.f);
      if (k < ns) v[k] = ns > 1 ? make_float2(tc::ld_cluster_f32(at, k), tc::ld_cluster_f32(at + 4, k)) : sml[tid];
      mx = fmaxf(mx, v[k].x);
    }
#pragma unroll
    for (int k = 0; k < MAX_SLICES; ++k) {
      v[k].x = v[k].y > 0.f ? expf(v[k].x - mx) : 0.f;
      l += v[k].x * v[k].y;
    }
#pragma unroll
    for (int k = 0; k < MAX_SLICES; ++k)
      if (k < ns) wt[k * 16 + tid] = v[k].x / l;
  }
  __syncthreads();
  const int share = (a.R + ns - 1) / ns, c_lo = split * share, c_hi = min(a.R, c_lo + share);
  // a warp takes heads `warp` and `warp + 8`: all remote loads of both are issued before the first use
  for (int col = c_lo + lane; col < c_hi; col += 32) {
    float p[2][MAX_SLICES];
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const uint32_t at = tc::smem_u32(so + (warp + 8 * x) * ldo + col);
#pragma unroll
      for (int k = 0; k < MAX_SLICES; ++k) p[x][k] = k < ns ? (ns > 1 ? tc::ld_cluster_f32(at, k) : so[(warp + 8 * x) * ldo + col]) : 0.f;
    }
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int r = warp + 8 * x;
      float v = 0.f;
#pragma unroll
      for (int k = 0; k < MAX_SLICES; ++k)
        if (k < ns) v += p[x][k] * wt[k * 16 + r];
      if (h0 + r < a.H) sc.o[(m * a.H + h0 + r) * a.R + col] = v;
    }
  }
  if (ns > 1) tc::cluster_sync_all();  // nobody leaves while another CTA may read its shared memory
}

// out[m, h, e] = Wuv[h, e] . o[m, h]: eight warps, two value rows each.  The rows of Wuv are fetched
// before the dependency wait and stay in registers (R <= 512) for all tokens.
__global__ void __launch_bounds__(256) k_latent_out(LatentArgs a, DecodeScratch s) {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, e0 = blockIdx.y * 16 + warp * 2;
  const __nv_bfloat16* uv = (const __nv_bfloat16*)a.uv + (int64_t)h * a.dv * a.R;
  const bool even = (a.R & 1) == 0;
  __nv_bfloat162 w[2][8];
#pragma unroll
  for (int y = 0; y < 2; ++y)
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const int i = 2 * lane + 64 * k;
      w[y][k] = __floats2bfloat162_rn(0.f, 0.f);
      if (e0 + y < a.dv && i < a.R) {
        const __nv_bfloat16* p = uv + (int64_t)(e0 + y) * a.R + i;
        if (even) w[y][k] = *(const __nv_bfloat162*)p;
        else w[y][k] = __nv_bfloat162(p[0], i + 1 < a.R ? p[1] : __float2bfloat16_rn(0.f));
      }
    }
  asm volatile("griddepcontrol.wait;" ::: "memory");
  for (int64_t m = blockIdx.z; m < a.rows.M; m += gridDim.z) {
    const float* o = s.o + (m * a.H + h) * a.R;
    float2 v[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) {
      const int i = 2 * lane + 64 * k;
      v[k] = make_float2(0.f, 0.f);
      if (i < a.R) {
        if (even) v[k] = *(const float2*)(o + i);
        else v[k] = make_float2(o[i], i + 1 < a.R ? o[i + 1] : 0.f);
      }
    }
    float acc[2] = {0.f, 0.f};
#pragma unroll
    for (int k = 0; k < 8; ++k)
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const float2 f = __bfloat1622float2(w[y][k]);
        acc[y] += v[k].x * f.x + v[k].y * f.y;
      }
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      acc[y] = warp_sum(acc[y]);
      if (lane == 0 && e0 + y < a.dv) ((__nv_bfloat16*)a.att)[m * a.ld_att + (int64_t)h * a.Do + e0 + y] = __float2bfloat16_rn(acc[y]);
    }
  }
}

int pick_nt(int R) { return R <= 128 ? 2 : R <= 256 ? 4 : R <= 512 ? 8 : 0; }
int row_pitch(const LatentArgs& a) { return std::max((int)(a.Lw + 15) / 16 * 16, pick_nt(a.R) * 64) + 8; }
size_t dec_smem(int ldk) { return (size_t)(16 + 2 * LD_KT) * ldk * 2 + 16 * 72 * 2 + 256 * 4; }  // (the merge fits over the tiles)

// context slices: enough blocks for every SM, at most about one tile each at full context
int pick_splits(const LatentArgs& a, int64_t M) {
  const int64_t base = M * ((a.H + 15) / 16);
  int s = 1;
  while (s < MAX_SLICES && base * (s * 2) <= 2 * 148 && (int64_t)s * LD_KT < a.Tmax) s *= 2;
  return s;
}

template <int NT>
int launch_dec(cg_ctx* c, const LatentArgs& a, const DecodeScratch& s) {
  const int ldk = row_pitch(a);
  const size_t smem = dec_smem(ldk);
  static PerDeviceSize configured_on;
  size_t& configured = configured_on.at(c->core->device);
  if (smem > configured) {
    CG_CUDA(c, cudaFuncSetAttribute(k_latent_dec<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = smem;
  }
  dim3 grid((unsigned)a.rows.M, (unsigned)((a.H + 15) / 16), (unsigned)s.splits);
  CG_CUDA(c, launch_kernel(c, k_latent_dec<NT>, grid, dim3(256), smem, s.splits, a, s, ldk));
  CG_LAUNCHED(c);
  return CG_OK;
}

size_t up16b(size_t n) { return (n + 15) / 16 * 16; }

}  // namespace

bool latent_decode_supported(int d, int R, int64_t Lw) {
  const int nt = pick_nt(R);
  if (!nt || Lw % 16 || d > 224) return false;
  return dec_smem(std::max((int)Lw, nt * 64) + 8) <= 227 * 1024;
}

size_t latent_decode_scratch(const LatentArgs& a, int64_t M) {
  const size_t n = (size_t)M * a.H;
  return up16b(n * a.Lw * 2) + n * a.R * 4;
}

int k_launch_latent_decode(cg_ctx* c, const LatentArgs& a, void* scratch) {
  const int64_t M = a.rows.M;
  if (M == 0) return CG_OK;
  DecodeScratch s;
  s.splits = pick_splits(a, M);
  const size_t n = (size_t)M * a.H;
  s.qa = (__nv_bfloat16*)scratch;
  s.o = (float*)((char*)scratch + up16b(n * a.Lw * 2));
  const int cb = (a.R + 63) / 64;
  const size_t sm1 = std::max<size_t>((size_t)(8 * 256 + 8 * a.d) * 4 + (size_t)a.d * 128, 128);
  CG_CUDA(c, launch_kernel(c, k_latent_absorb, dim3((unsigned)(a.H * cb + M)), dim3(256), sm1, 1, a, s, cb));
  CG_LAUNCHED(c);
  switch (pick_nt(a.R)) {
    case 2: CG_TRY(launch_dec<2>(c, a, s)); break;
    case 4: CG_TRY(launch_dec<4>(c, a, s)); break;
    default: CG_TRY(launch_dec<8>(c, a, s)); break;
  }
  const int eb = (a.dv + 15) / 16;
  const int mz = (int)std::min<int64_t>(M, std::max<int64_t>(1, 4 * 148 / std::max(1, a.H * eb)));
  CG_CUDA(c, launch_kernel(c, k_latent_out, dim3((unsigned)a.H, (unsigned)eb, (unsigned)mz), dim3(256), 0, 1, a, s));
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace cg
