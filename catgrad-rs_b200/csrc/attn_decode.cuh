// attn_decode.cuh — the attention block of a decode step for one (row, kv head, context slice),
// as a device function shared by the stand-alone kernel (attn_decode.cu: one CTA per item, the
// slices of a pair forming a thread-block cluster) and the resident decode kernel
// (decode_resident.cu: 128 threads of a resident CTA work through a list of items).
//
// The caller supplies an environment:
//   tid()            0..127, the thread's index among the 128 threads that run the item
//   sync_cta()       barrier among those 128 threads
//   sync_group()     barrier among the CTAs that hold the slices of one (row, kv head),
//                    including a barrier among each CTA's own 128 threads
//   cluster_rank(s)  cluster rank of the CTA that holds slice s
//   kPush / landing()  kPush: the slices' partial results are PUSHED into a landing area (of
//                    attn_dec_landing_bytes(), shared memory that nothing else uses) of the CTA that
//                    finishes them, so one group barrier suffices and nobody waits before leaving;
//                    otherwise the finishing CTA reads the partials where they lie (two barriers)
//   kRows            the item is a row of AttnDecArgs::rows: its own slot and position, neighbouring pairs
//                    rotated, norms over all heads at once, a sink
//   settle(pos)      called once the first K/V tiles have been requested with a position that may
//                    be one step old: waits for whatever the caller's inputs depend on and returns
//                    the position to use (cached keys never change, so an early request is either
//                    right or is repeated)
#pragma once

#include "kernels.h"
#include "mma.cuh"

namespace cg {

constexpr int ATTN_MAX_REP = 8;  // query heads per kv head: rows 0..7 of the 16-row MMA tile

__device__ __forceinline__ float attn_tanh_sig(float x) { return 2.f / (1.f + __expf(-2.f * x)) - 1.f; }
__device__ __forceinline__ float attn_ld_dsmem(uint32_t local_addr, uint32_t rank) {
  uint32_t remote;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local_addr), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
  return v;
}

// shared memory one item needs
template <int D>
__host__ __device__ constexpr size_t attn_dec_smem_bytes() {
  return (size_t)(16 * (D + 8) + 8 * (D > 128 ? 16 : 32) * (D + 8)) * 2 + (size_t)(2 * D + 8 * ATTN_MAX_REP + 16) * 4;
}

// landing area of the push form: {max, sum} per source slice and head, then per source slice the
// output values the CTA finishes (at most 8 slices; up to rep * D / 128 + 8 blocks of 128 values)
__host__ __device__ constexpr size_t attn_dec_landing_bytes() { return (size_t)(8 * ATTN_MAX_REP * 2 + (16 + 8) * 128) * 4; }

// KT = keys per warp tile: 32, or 16 for head size 256 so that a CTA's tiles fit a third of an
// SM's shared memory.
template <int D, class Env>
__device__ __forceinline__ void attn_dec_item(const AttnDecArgs& a, float scale, int kvh, int64_t b, int split, int64_t pos_early,
                                              uint8_t* smem, Env& env) {
  constexpr int KT = D > 128 ? 16 : 32;
  constexpr int MAX_REP = ATTN_MAX_REP;
  constexpr int LD = D + 8;     // padded rows: conflict-free ldmatrix
  constexpr int CH = D / 8;     // 16-byte chunks per row
  constexpr int NT = D / 8;     // output n-tiles
  __nv_bfloat16* qt = (__nv_bfloat16*)smem;              // [16][LD] query heads (rows >= rep are zero)
  __nv_bfloat16* kt = qt + 16 * LD;                      // [4 warps][KT][LD] key tiles
  __nv_bfloat16* vt = kt + 4 * KT * LD;                  // [4 warps][KT][LD] value tiles
  float* fl = (float*)(vt + 4 * KT * LD);
  float* knew = fl;                                      // [D] the new key (bf16-rounded)
  float* vnew = knew + D;                                // [D]
  float* red_m = vnew + D;                               // [4][MAX_REP]
  float* red_l = red_m + 4 * MAX_REP;                    // [4][MAX_REP]
  float* hsq = red_l + 4 * MAX_REP;                      // [MAX_REP + 1] per-head rms (norm), padded to 16
  float* red_o = (float*)kt;                             // [4][MAX_REP][D] f32, reuses the tiles after the loop

  const int tid = env.tid(), warp = tid >> 5, lane = tid & 31;
  const int rep = a.nh / a.nkv;
  const int half = D / 2;
  // pos: position of the new token = number of cached keys.  The projected row is read with
  // L2 loads: in the resident kernel another CTA wrote it earlier in the same launch.
  int64_t place = b;
  if constexpr (Env::kRows) place = a.rows.slot[b];
  __nv_bfloat16* kbase = a.k_cache + ((place * a.nkv + kvh) * a.Tmax) * (int64_t)D;
  __nv_bfloat16* vbase = a.v_cache + ((place * a.nkv + kvh) * a.Tmax) * (int64_t)D;

  // The visible cached keys are the kf kept first ones and [lo, pos); [t0, t1) is this CTA's slice of
  // their sequence.
  int64_t pos = pos_early, t0 = 0, t1 = 0, lo = 0, kf = 0;
  auto plan = [&]() {
    lo = a.window > 0 ? max((int64_t)0, pos - a.window + 1) : 0;
    if constexpr (Env::kRows) kf = min(a.keep_first, lo);
    const int64_t span = kf + pos - lo;
    int64_t per = (span + a.splits - 1) / a.splits;
    per = (per + KT - 1) / KT * KT;
    t0 = split * per;
    t1 = min(span, t0 + per);
  };
  plan();

  __nv_bfloat16* kw = kt + (size_t)warp * KT * LD;
  __nv_bfloat16* vw = vt + (size_t)warp * KT * LD;
  const uint32_t kw_u = (uint32_t)__cvta_generic_to_shared(kw);
  const uint32_t vw_u = (uint32_t)__cvta_generic_to_shared(vw);
  const uint32_t qt_u = (uint32_t)__cvta_generic_to_shared(qt);

  // request the first chunk of this warp now: it does not depend on q
  auto request = [&](int64_t c0) {
    // KT rows x CH chunks, 8 (or more) lanes per row: fully coalesced 16-byte copies
    for (int i = lane; i < KT * CH; i += 32) {
      const int r = i / CH, ch = i - r * CH;
      const int64_t key = c0 + r;
      const bool ok = key < t1;
      int64_t kc = ok ? key : t0;
      if (kc >= kf) kc += lo - kf;
      cp_async16(kw_u + (uint32_t)(r * LD + ch * 8) * 2u, kbase + kc * (int64_t)D + ch * 8, ok ? 16 : 0);
      cp_async16(vw_u + (uint32_t)(r * LD + ch * 8) * 2u, vbase + kc * (int64_t)D + ch * 8, ok ? 16 : 0);
    }
  };
  int64_t c0 = t0 + warp * KT;
  if (c0 < t1) request(c0);
  {
    const int64_t pos_now = env.settle(pos);
    if (pos_now != pos) {  // the early position was stale: let the copies land, then ask again
      cp_async_wait_all();
      __syncwarp();
      pos = pos_now;
      plan();
      c0 = t0 + warp * KT;
      if (c0 < t1) request(c0);
    }
  }

  // ---- 1. q, k, v of the new token ----
  const int heads = a.nh + 2 * a.nkv;
  int64_t ld_row = (int64_t)heads * D, ld_out = (int64_t)a.nh * D;
  if constexpr (Env::kRows) {
    if (a.ld_qkv) ld_row = a.ld_qkv;
    if (a.ld_out) ld_out = a.ld_out;
  }
  const float* row = a.qkv + b * ld_row;
  const float* qsrc = row + (int64_t)kvh * rep * D;
  const float* ksrc = row + ((int64_t)a.nh + kvh) * D;
  const float* vsrc = row + ((int64_t)a.nh + a.nkv + kvh) * D;
  if constexpr (Env::kRows) {
    if (a.q_gamma) {
      // norms over all query heads and over all key heads: hsq[0], hsq[1] receive the factors
      float ss[2] = {0.f, 0.f};
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        const float4* src = (const float4*)(row + (part ? (int64_t)a.nh * D : 0));
        const int n = (part ? a.nkv : a.nh) * D / 4;
#pragma unroll 4
        for (int i = tid; i < n; i += 128) {
          const float4 v = __ldcg(src + i);
          ss[part] += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
#pragma unroll
        for (int o = 16; o; o >>= 1) ss[part] += __shfl_xor_sync(0xffffffffu, ss[part], o);
        if (lane == 0) red_m[part * 4 + warp] = ss[part];
      }
      env.sync_cta();
      if (tid < 2) {
        const float* r = red_m + tid * 4;
        hsq[tid] = 1.f / sqrtf(((r[0] + r[1]) + (r[2] + r[3])) / (float)((tid ? a.nkv : a.nh) * a.norm_dim) + a.norm_eps);
      }
      env.sync_cta();
    } else if (a.head_norm) {
      // norms per head: hsq[h] of the query heads, hsq[rep] of the key head
      for (int h = warp; h <= rep; h += 4) {
        const float* src = h < rep ? qsrc + h * D : ksrc;
        float ss = 0.f;
        for (int e = lane; e < D; e += 32) { const float v = __ldcg(src + e); ss += v * v; }
#pragma unroll
        for (int o = 16; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if (lane == 0) hsq[h] = 1.f / sqrtf(ss / (float)a.norm_dim + a.norm_eps);
      }
      env.sync_cta();
    }
    // neighbouring components (2 j, 2 j + 1) of the first rot_dims turn together
    const int rh = a.rot_dims / 2;
    const float temp = a.q_temp ? a.q_temp[pos] : 1.f;
    const float* ct = a.cos_t + pos * rh;
    const float* st = a.sin_t + pos * rh;
    for (int i = tid; i < 16 * half; i += 128) {
      const int h = i / half, j = i - h * half;
      float x1 = 0.f, x2 = 0.f;
      if (h < rep) {
        const float2 x = __ldcg((const float2*)(qsrc + h * D) + j);
        x1 = x.x; x2 = x.y;
        if (a.q_gamma) {
          const float2 g = *((const float2*)(a.q_gamma + (kvh * rep + h) * D) + j);
          x1 *= hsq[0] * g.x; x2 *= hsq[0] * g.y;
        } else if (a.head_norm) {
          x1 *= hsq[h]; x2 *= hsq[h];
        }
        if (j < rh) {
          const float cs = ct[j], sn = st[j], t = x1;
          x1 = cs * t - sn * x2;
          x2 = cs * x2 + sn * t;
        }
        x1 *= temp; x2 *= temp;
      }
      *(__nv_bfloat162*)(qt + h * LD + 2 * j) = __floats2bfloat162_rn(x1, x2);
    }
    for (int j = tid; j < half; j += 128) {
      const float2 x = __ldcg((const float2*)ksrc + j), v = __ldcg((const float2*)vsrc + j);
      float x1 = x.x, x2 = x.y;
      if (a.q_gamma) {
        const float2 g = *((const float2*)(a.k_gamma + kvh * D) + j);
        x1 *= hsq[1] * g.x; x2 *= hsq[1] * g.y;
      } else if (a.head_norm) {
        x1 *= hsq[rep]; x2 *= hsq[rep];
      }
      if (j < rh) {
        const float cs = ct[j], sn = st[j], t = x1;
        x1 = cs * t - sn * x2;
        x2 = cs * x2 + sn * t;
      }
      const __nv_bfloat162 kk = __floats2bfloat162_rn(x1, x2), vv = __floats2bfloat162_rn(v.x, v.y);
      knew[2 * j] = __low2float(kk); knew[2 * j + 1] = __high2float(kk);
      vnew[2 * j] = __low2float(vv); vnew[2 * j + 1] = __high2float(vv);
      if (split == 0) {  // append to the cache for the following steps
        *(__nv_bfloat162*)(kbase + pos * D + 2 * j) = kk;
        *(__nv_bfloat162*)(vbase + pos * D + 2 * j) = vv;
      }
    }
    env.sync_cta();
  } else {
  if (a.q_gamma) {
    // per-head RMSNorm over d for the rep query heads and the key head
    for (int h = warp; h <= rep; h += 4) {
      const float* src = h < rep ? qsrc + h * D : ksrc;
      float ss = 0.f;
      for (int e = lane; e < D; e += 32) { const float v = __ldcg(src + e); ss += v * v; }
#pragma unroll
      for (int o = 16; o; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (lane == 0) hsq[h] = sqrtf(ss / (float)D + a.norm_eps);
    }
    env.sync_cta();
  }
  for (int i = tid; i < 16 * half; i += 128) {
    const int h = i / half, j = i - h * half;
    if (h < rep) {
      float x1 = __ldcg(qsrc + h * D + j), x2 = __ldcg(qsrc + h * D + j + half);
      if (a.q_gamma) {
        const float g1 = a.norm_plus_one ? 1.f + a.q_gamma[j] : a.q_gamma[j];
        const float g2 = a.norm_plus_one ? 1.f + a.q_gamma[j + half] : a.q_gamma[j + half];
        x1 = x1 / hsq[h] * g1;
        x2 = x2 / hsq[h] * g2;
      }
      const float cs = a.cos_t[pos * half + j], sn = a.sin_t[pos * half + j];
      qt[h * LD + j] = __float2bfloat16_rn(cs * x1 - sn * x2);
      qt[h * LD + j + half] = __float2bfloat16_rn(cs * x2 + sn * x1);
    } else {
      qt[h * LD + j] = __float2bfloat16_rn(0.f);
      qt[h * LD + j + half] = __float2bfloat16_rn(0.f);
    }
  }
  for (int j = tid; j < half; j += 128) {
    float x1 = __ldcg(ksrc + j), x2 = __ldcg(ksrc + j + half);
    if (a.q_gamma) {
      const float g1 = a.norm_plus_one ? 1.f + a.k_gamma[j] : a.k_gamma[j];
      const float g2 = a.norm_plus_one ? 1.f + a.k_gamma[j + half] : a.k_gamma[j + half];
      x1 = x1 / hsq[rep] * g1;
      x2 = x2 / hsq[rep] * g2;
    }
    const float cs = a.cos_t[pos * half + j], sn = a.sin_t[pos * half + j];
    const __nv_bfloat16 k1 = __float2bfloat16_rn(cs * x1 - sn * x2), k2 = __float2bfloat16_rn(cs * x2 + sn * x1);
    const __nv_bfloat16 v1 = __float2bfloat16_rn(__ldcg(vsrc + j)), v2 = __float2bfloat16_rn(__ldcg(vsrc + j + half));
    knew[j] = __bfloat162float(k1);
    knew[j + half] = __bfloat162float(k2);
    vnew[j] = __bfloat162float(v1);
    vnew[j + half] = __bfloat162float(v2);
    if (split == 0) {  // append to the cache for the following steps
      kbase[pos * D + j] = k1;
      kbase[pos * D + j + half] = k2;
      vbase[pos * D + j] = v1;
      vbase[pos * D + j + half] = v2;
    }
  }
  env.sync_cta();
  }

  // ---- 2. this warp's chunks of 32 keys: S = Q K^T, online softmax, O += P V ----
  // A thread owns head r = lane / 4 (rows 8..15 of the MMA tile are padding) and, per 8-key
  // or 8-column tile, the two columns 2 * (lane % 4) + {0, 1}.
  const int hr = lane >> 2, cq = (lane & 3) * 2;
  const float* bias = nullptr;
  if constexpr (Env::kRows)
    if (a.bias && hr < rep) bias = a.bias + (int64_t)(kvh * rep + hr) * a.ld_bias;
  float m = -INFINITY, l = 0.f;
  float o[NT][4];
#pragma unroll
  for (int j = 0; j < NT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;

  // slice 0, warp 0 also owns the new token: one more chunk whose only live key is row 0
  const bool owns_new = split == 0 && warp == 0;
  bool do_new = false;
  while (true) {
    int64_t limit;  // live keys of this chunk are [c0, limit)
    if (c0 < t1) {
      limit = t1;
      cp_async_wait_all();
      __syncwarp();
    } else if (owns_new && !do_new) {
      do_new = true;
      // build the one-row chunk in the tiles
      for (int e = lane; e < D; e += 32) {
        kw[e] = __float2bfloat16_rn(knew[e]);
        vw[e] = __float2bfloat16_rn(vnew[e]);
      }
      for (int i = lane; i < (KT - 1) * CH; i += 32) {
        const int r = 1 + i / CH, ch = i % CH;
        *(uint4*)(vw + r * LD + ch * 8) = make_uint4(0u, 0u, 0u, 0u);  // p = 0 times NaN garbage must not happen
        *(uint4*)(kw + r * LD + ch * 8) = make_uint4(0u, 0u, 0u, 0u);
      }
      __syncwarp();
      limit = 1;  // in units relative to a chunk start of 0
    } else {
      break;
    }
    const int64_t cbase = do_new ? 0 : c0;

    float s[KT / 8][4];
#pragma unroll
    for (int j = 0; j < KT / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < D / 16; ++kk) {
      uint32_t a0, a1, a2, a3;
      {
        const int r = (lane & 7) + 8 * ((lane >> 3) & 1);
        const int col = kk * 16 + 8 * (lane >> 4);
        ldsm_x4(qt_u + (uint32_t)(r * LD + col) * 2u, a0, a1, a2, a3);
      }
#pragma unroll
      for (int j = 0; j < KT / 8; j += 2) {
        uint32_t b0, b1, b2, b3;
        const int key = j * 8 + (lane & 7) + 8 * (lane >> 4);
        const int col = kk * 16 + 8 * ((lane >> 3) & 1);
        ldsm_x4(kw_u + (uint32_t)(key * LD + col) * 2u, b0, b1, b2, b3);
        mma_bf16(s[j], a0, a1, a2, a3, b0, b1);
        mma_bf16(s[j + 1], a0, a1, a2, a3, b2, b3);
      }
    }
    // scale, soft-cap, mask; this head's maximum over the chunk
    float mx = -INFINITY;
#pragma unroll
    for (int j = 0; j < KT / 8; ++j) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float v = s[j][e] * scale;
        if (a.softcap > 0.f) v = a.softcap * attn_tanh_sig(v / a.softcap);
        const bool keep = cbase + j * 8 + cq + e < limit;
        if constexpr (Env::kRows)
          if (bias && keep && !do_new) {   // (at the new token itself the distance is 0, and so is what is taken off)
            const int64_t i = cbase + j * 8 + cq + e;
            v -= bias[pos - (i < kf ? i : i - kf + lo)];
          }
        v = keep ? v : -INFINITY;
        s[j][e] = v;
        mx = fmaxf(mx, v);
      }
    }
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
    mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
    const float mnew = fmaxf(m, mx);  // finite: the first key of every chunk is live
    const float corr = __expf(m - mnew);
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < KT / 8; ++j) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float p = __expf(s[j][e] - mnew);
        s[j][e] = p;
        sum += p;
      }
    }
    sum += __shfl_xor_sync(0xffffffffu, sum, 1);
    sum += __shfl_xor_sync(0xffffffffu, sum, 2);
    l = l * corr + sum;
    m = mnew;
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      o[j][0] *= corr;
      o[j][1] *= corr;
    }
    // O += P V; rows 8..15 of P are zero
#pragma unroll
    for (int kk = 0; kk < KT / 16; ++kk) {
      const uint32_t a0 = pack_bf16(s[2 * kk][0], s[2 * kk][1]);
      const uint32_t a2 = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
#pragma unroll
      for (int j = 0; j < NT; j += 2) {
        uint32_t b0, b1, b2, b3;
        const int key = kk * 16 + (lane & 7) + 8 * ((lane >> 3) & 1);
        const int col = j * 8 + 8 * (lane >> 4);
        ldsm_x4_t(vw_u + (uint32_t)(key * LD + col) * 2u, b0, b1, b2, b3);
        mma_bf16(o[j], a0, 0u, a2, 0u, b0, b1);
        mma_bf16(o[j + 1], a0, 0u, a2, 0u, b2, b3);
      }
    }
    __syncwarp();
    if (do_new) break;
    c0 += 4 * KT;
    if (c0 < t1) request(c0);
  }

  // ---- 3. merge the four warps in this CTA, then the slices across the cluster ----
  env.sync_cta();  // all tiles are dead: reuse their space
  if (hr < rep) {
    if ((lane & 3) == 0) { red_m[warp * MAX_REP + hr] = m; red_l[warp * MAX_REP + hr] = l; }
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      red_o[(warp * MAX_REP + hr) * D + j * 8 + cq] = o[j][0];
      red_o[(warp * MAX_REP + hr) * D + j * 8 + cq + 1] = o[j][1];
    }
  }
  env.sync_cta();
  // this slice's partial: part[r] = {max, sum}, part_o[r][e], left in shared memory for the cluster
  float* part_ml = (float*)vt;                 // [MAX_REP][2]
  float* part_o = part_ml + 2 * MAX_REP;       // [MAX_REP][D]
  const int S = a.splits;
  // the merged output oo over the merged sum ll of exp(score - mm), which the sink joins, gated and scaled
  auto finished = [&](int r, int e, float mm, float ll, float oo) {
    if constexpr (Env::kRows) {
      oo *= a.out_scale;
      if (a.gate) oo *= 1.f / (1.f + __expf(-__ldcg(a.gate + b * a.ld_gate + (a.wide_gate ? (kvh * rep + r) * D + e : kvh * rep + r))));
      if (a.sink) {
        const float sk = a.sink[kvh * rep + r], top = fmaxf(mm, sk);
        const float f = __expf(mm - top);
        return oo * f / (ll * f + __expf(sk - top));
      }
    }
    return ll > 0.f ? oo / ll : 0.f;
  };
  const bool push = Env::kPush && a.push_merge && S > 1;
  // push form: output i is finished by slice (i / 128) % S, as its block number (i / 128) / S
  const int kmax = (rep * D + 128 * S - 1) / (128 * S);
  float* land_ml = nullptr;   // [8][MAX_REP][2]
  float* land_o = nullptr;    // [S][kmax][128]
  uint32_t land_u = 0;
  if (push) {
    land_ml = env.landing();
    land_o = land_ml + 8 * MAX_REP * 2;
    land_u = (uint32_t)__cvta_generic_to_shared(land_ml);
  }
  auto st_remote = [&](uint32_t local_addr, uint32_t rank, float v) {
    uint32_t remote;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(local_addr), "r"(rank));
    asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(remote), "f"(v) : "memory");
  };
  for (int i = tid; i < rep * D; i += 128) {
    const int r = i / D, e = i - r * D;
    float mm = -INFINITY;
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, red_m[w * MAX_REP + r]);
    float ll = 0.f, oo = 0.f;
    for (int w = 0; w < 4; ++w) {
      const float mw = red_m[w * MAX_REP + r];
      const float f = mw == -INFINITY ? 0.f : __expf(mw - mm);
      ll += red_l[w * MAX_REP + r] * f;
      oo += red_o[(w * MAX_REP + r) * D + e] * f;
    }
    if (push) {
      const int blk = i >> 7;
      st_remote(land_u + (uint32_t)(8 * MAX_REP * 2 + ((split * kmax + blk / S) << 7) + (i & 127)) * 4u, env.cluster_rank(blk % S), oo);
      if (e == 0)
        for (int s = 0; s < S; ++s) {
          st_remote(land_u + (uint32_t)((split * MAX_REP + r) * 2) * 4u, env.cluster_rank(s), mm);
          st_remote(land_u + (uint32_t)((split * MAX_REP + r) * 2 + 1) * 4u, env.cluster_rank(s), ll);
        }
      continue;
    }
    if (e == 0) { part_ml[2 * r] = mm; part_ml[2 * r + 1] = ll; }
    part_o[r * D + e] = oo;
  }
  if (push) {
    // one barrier: every slice's pushes are visible after it and nobody touches another CTA's
    // shared memory again
    env.sync_group();
    int k = 0;
    for (int i = tid + 128 * split; i < rep * D; i += 128 * S, ++k) {
      const int r = i / D;
      float ms[8], ls[8], os[8];
#pragma unroll
      for (int s = 0; s < 8; ++s) {
        const bool in = s < S;
        ms[s] = in ? land_ml[(s * MAX_REP + r) * 2] : -INFINITY;
        ls[s] = in ? land_ml[(s * MAX_REP + r) * 2 + 1] : 0.f;
        os[s] = in ? land_o[((s * kmax + k) << 7) + tid] : 0.f;
      }
      float mm = -INFINITY;
#pragma unroll
      for (int s = 0; s < 8; ++s) mm = fmaxf(mm, ms[s]);
      float ll = 0.f, oo = 0.f;
#pragma unroll
      for (int s = 0; s < 8; ++s) {
        const float f = ms[s] == -INFINITY ? 0.f : __expf(ms[s] - mm);
        ll += ls[s] * f;
        oo += os[s] * f;
      }
      a.out[b * ld_out + (kvh * rep + r) * (int64_t)D + (i - r * D)] = __float2bfloat16_rn(finished(r, i - r * D, mm, ll, oo));
    }
    return;
  }
  if (S == 1) {
    env.sync_cta();
    for (int i = tid; i < rep * D; i += 128) {
      const int r = i / D, e = i - r * D;
      const float ll = part_ml[2 * r + 1];
      a.out[b * ld_out + (kvh * rep + r) * (int64_t)D + e] = __float2bfloat16_rn(finished(r, e, part_ml[2 * r], ll, part_o[i]));
    }
    env.sync_cta();  // the partials are read: the next item of a resident CTA may reuse the space
    return;
  }
  // the slices of one (row, kv head) are one thread-block cluster: merge over distributed
  // shared memory, each CTA finishing an interleaved share of the outputs
  env.sync_group();
  const uint32_t ml_u = (uint32_t)__cvta_generic_to_shared(part_ml);
  const uint32_t po_u = (uint32_t)__cvta_generic_to_shared(part_o);
  for (int i = tid + 128 * split; i < rep * D; i += 128 * S) {
    const int r = i / D;
    // all remote loads first (their latencies overlap), then the arithmetic; S <= 8
    float ms[8], ls[8], os[8];
#pragma unroll
    for (int s = 0; s < 8; ++s) {
      const bool in = s < S;
      ms[s] = in ? attn_ld_dsmem(ml_u + (uint32_t)(2 * r) * 4u, env.cluster_rank(s)) : -INFINITY;
      ls[s] = in ? attn_ld_dsmem(ml_u + (uint32_t)(2 * r + 1) * 4u, env.cluster_rank(s)) : 0.f;
      os[s] = in ? attn_ld_dsmem(po_u + (uint32_t)i * 4u, env.cluster_rank(s)) : 0.f;
    }
    float mm = -INFINITY;
#pragma unroll
    for (int s = 0; s < 8; ++s) mm = fmaxf(mm, ms[s]);
    float ll = 0.f, oo = 0.f;
#pragma unroll
    for (int s = 0; s < 8; ++s) {
      const float f = ms[s] == -INFINITY ? 0.f : __expf(ms[s] - mm);
      ll += ls[s] * f;
      oo += os[s] * f;
    }
    a.out[b * ld_out + (kvh * rep + r) * (int64_t)D + (i - r * D)] = __float2bfloat16_rn(finished(r, i - r * D, mm, ll, oo));
  }
  // nobody leaves while a peer may still read its shared memory
  env.sync_group();
}

}  // namespace cg
