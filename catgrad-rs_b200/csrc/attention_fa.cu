// attention_fa.cu — causal prefill attention on the Blackwell tensor cores (tcgen05 + TMEM),
// for head sizes 64 and 128 without soft-cap.
//
// Same mathematics as attention.cu (catgrad-llm/src/models/llama.rs:97-108 after repeat_kv,
// catgrad-llm/src/helpers.rs:147-161, as an online-softmax pass over key tiles); what changes
// is where the two matrix products run:
//
//   warp 0      TMA: the 128-query tile once, then 128-key K and V tiles through two
//               shared-memory buffers each
//   warp 1      one lane issues S = Q K^T (128 x 128, f32 in TMEM, two S buffers so the next
//               tile's scores are computed while this tile's softmax runs) and O_t = P V
//               (128 x D, f32 in TMEM)
//   warps 2-5   one thread per query row (TMEM lane = row, so row maxima and sums need no
//               shuffles): read the score row from TMEM, mask, exponentiate, write P as bf16
//               into shared memory in the 128-byte-swizzled k-major layout the MMA reads,
//               then fold O_t into the row's running output kept in registers
//
// V is consumed as it lies in the cache ([keys, D], D contiguous): for P V it is the MMA's B
// operand with the "MN-major" layout bit, i.e. no transposed copy of V exists anywhere.
//
// Every mbarrier wait is bounded; on expiry the kernel raises the context's error word, all
// roles leave their loops, TMEM is freed and the kernel returns.
#include <algorithm>

#include "act.cuh"
#include "kernels.h"
#include "tc_common.cuh"

namespace cg {

namespace {

using namespace tc;

constexpr int FA_BQ = 128;
constexpr float LOG2E = 1.4426950408889634f;

struct FaArgs {
  __nv_bfloat16* out;  // [B * S, nh D]
  int64_t S, pos0, Tmax;
  int nh, nkv;
  int token_major;     // keys and values lie token after token, the heads side by side
  float scale_log2e;   // score factor (1 / sqrt(D)) * log2(e)
  int64_t window;      // 0 = none
  int64_t keep;        // with a window: first positions that stay visible
  const float* sink;   // [nh] or null
  const float* gate;   // [tokens, ld_gate] or null: sigmoid(gate) multiplies a head's output, as out_scale does
  int64_t ld_gate, ld_out;
  int wide_gate;       // a gate per value instead of one per head
  const float* bias;   // EXTRA: bias[h * ld_bias + distance] is taken off the scores
  int64_t ld_bias;
  float out_scale;
  RowsDev rows;        // rows of unequal length (rows.rows > 0)
  int32_t* err;
};

// B operand stored [k rows][n contiguous] ("MN-major") in 128-byte-swizzled boxes of
// [rows, 64 elements]: 64-element chunks along n are `chunk_bytes` apart, groups of 8 k rows
// 1024 bytes apart.
__device__ __forceinline__ uint64_t umma_desc_mn(uint32_t saddr, uint32_t chunk_bytes) {
  uint64_t d = 0;
  d |= (uint64_t)((saddr & 0x3FFFFu) >> 4);
  d |= (uint64_t)((chunk_bytes >> 4) & 0x3FFFu) << 16;  // leading byte offset: next 64-element chunk along n
  d |= (uint64_t)(1024 >> 4) << 32;                     // stride byte offset: next group of 8 k rows
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;                               // SWIZZLE_128B
  return d;
}

// the lowest n bits, n of any size
__device__ __forceinline__ uint32_t bits_below(int n) { return n <= 0 ? 0u : n >= 32 ? 0xffffffffu : (1u << n) - 1u; }

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// 32 consecutive TMEM columns of this thread's lane
__device__ __forceinline__ void tmem_ld32(uint32_t taddr, uint32_t* v) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
      "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
      : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]),
        "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]), "=r"(v[16]), "=r"(v[17]),
        "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), "=r"(v[23]), "=r"(v[24]), "=r"(v[25]), "=r"(v[26]),
        "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
      : "r"(taddr)
      : "memory");
}

// EXTRA: a gate per value (wide_gate), and a number per head and distance that is taken off the scores,
// monotone in the distance (bias null: none).  A tile's numbers,
// times -log2(e), lie in shared memory by ascending key, T[x] for key k0 + x - 127 against the tile's row 0 (row r
// reads T[127 - r + c]), in four copies shifted by one entry each, so that every row reads four keys at a
// time from the copy in which they are aligned.  A row's maximum is then an upper bound: the largest
// product less the smallest number of the tile.
template <int D, int FA_BK, bool EXTRA>
__global__ void __launch_bounds__(192, FA_BK == 64 ? 2 : 1)
k_attn_fa(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
          const __grid_constant__ CUtensorMap map_v, FaArgs p) {
  constexpr int SUB = D / 64;                       // 64-wide sub-tiles along the head dimension
  constexpr uint32_t BOX = 128 * 128;               // bytes of one [128 rows, 64 bf16] box (Q, P)
  constexpr uint32_t KBOX = FA_BK * 128;            // bytes of one [FA_BK keys, 64 bf16] box (K, V)
  constexpr uint32_t Q_BYTES = SUB * BOX, KV_BYTES = SUB * KBOX, P_BYTES = (FA_BK / 64) * BOX;
  constexpr uint32_t S_COLS = FA_BK;                // one score buffer
  constexpr uint32_t O_COL = 2 * S_COLS;            // O_t after the two score buffers
  constexpr uint32_t NCOLS = 2 * S_COLS + D <= 256 ? 256 : 512;  // two CTAs per SM share 512 columns

  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");

  extern __shared__ __align__(1024) uint8_t smem_raw[];
  const uint32_t raw = smem_u32(smem_raw);
  const uint32_t base = (raw + 1023u) & ~1023u;
  if (FA_BK == 64 && base != raw) {
    // the 64-key variant is sized without alignment slack (two CTAs must fit one SM)
    if (threadIdx.x == 0) *p.err = DEV_TIMEOUT;
    return;
  }
  const uint32_t sq = base, sk = sq + Q_BYTES, sv = sk + 2 * KV_BYTES, sp = sv + 2 * KV_BYTES;
  const uint32_t bars = sp + P_BYTES;
  uint8_t* gen = smem_raw + (base - raw);
  // barriers (8 bytes each)
  const uint32_t b_q_full = bars, b_k_full = bars + 8, b_v_full = bars + 24, b_k_empty = bars + 40, b_v_empty = bars + 56,
                 b_s_full = bars + 72, b_s_empty = bars + 88, b_p_full = bars + 104, b_p_empty = bars + 112,
                 b_o_full = bars + 120, b_o_empty = bars + 128, b_bias = bars + 136;
  volatile uint32_t* tmem_slot = (volatile uint32_t*)(gen + (bars - base) + 144);
  volatile int* cta_abort = (volatile int*)(gen + (bars - base) + 148);
  constexpr int BIAS_N = 127 + FA_BK + 1, BIAS_LD = BIAS_N + 8;  // (copies 8 banks apart)
  float* const bias_tab = (float*)(gen + (bars - base) + 160);   // [2][4][BIAS_LD]

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int qt = (int)gridDim.x - 1 - (int)blockIdx.x, h = blockIdx.y;  // longest tiles first
  // the row: its first packed token, its length, the position of its first token, its place in the cache
  int64_t b = blockIdx.z, tok0 = b * p.S, len = p.S, start_pos = p.pos0;
  if (p.rows.rows > 0) {
    const int row = (int)b;  // (the row tables are written in plain stream order before a prompt's kernels)
    tok0 = p.rows.start[row];
    len = p.rows.start[row + 1] - tok0;
    start_pos = row_pos0(p.rows, row);
    b = p.rows.slot[row];
  }
  const int kvh = h / (p.nh / p.nkv);
  const int64_t q0 = (int64_t)qt * FA_BQ;
  if (q0 >= len) return;  // uniform over the CTA, before anything is allocated
  const int64_t last_q = start_pos + std::min<int64_t>(len, q0 + FA_BQ) - 1;
  // key tiles: nk of kept first tokens, then from tile j0 on
  const int j0 = p.window > 0 ? (int)(std::max<int64_t>(0, start_pos + q0 - p.window + 1) / FA_BK) : 0;
  const int nk = (int)std::min<int64_t>(j0, (p.keep + FA_BK - 1) / FA_BK);
  const int nt = nk + (int)(last_q / FA_BK) + 1 - j0;
  auto tile_of = [&](int j) { return j < nk ? j : j0 + j - nk; };

  if (tid == 0) {
    mbar_init(b_q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(b_k_full + 8 * i, 1);
      mbar_init(b_v_full + 8 * i, 1);
      mbar_init(b_k_empty + 8 * i, 1);
      mbar_init(b_v_empty + 8 * i, 1);
      mbar_init(b_s_full + 8 * i, 1);
      mbar_init(b_s_empty + 8 * i, 128);
    }
    mbar_init(b_p_full, 128);
    mbar_init(b_p_empty, 1);
    mbar_init(b_o_full, 1);
    mbar_init(b_o_empty, 128);
    mbar_init(b_bias, 128);
    *cta_abort = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32((const void*)tmem_slot)),
                 "r"(NCOLS)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem_base = *tmem_slot;

  // q and the cache are written by the preceding kernels
  asm volatile("griddepcontrol.wait;" ::: "memory");

  if (warp == 0) {
    if (lane == 0) {
      const int qrow = (int)(tok0 + q0);
      mbar_expect_tx(b_q_full, Q_BYTES);
      for (int s = 0; s < SUB; ++s) tma_load_2d(sq + s * BOX, &map_q, h * D + s * 64, qrow, b_q_full);
      const int64_t kvrow0 = p.token_major ? b * p.Tmax : (b * p.nkv + kvh) * p.Tmax;
      const int kx = p.token_major ? kvh * D : 0;
      bool ok = true;
      for (int j = 0; j < nt && ok; ++j) {
        const uint32_t buf = (uint32_t)j & 1u, ph = ((uint32_t)j >> 1) & 1u;
        const int row = (int)(kvrow0 + (int64_t)tile_of(j) * FA_BK);
        if (j >= 2) {
          ok = mbar_wait(b_k_empty + 8 * buf, ph ^ 1u, cta_abort, p.err);
          if (!ok) break;
        }
        mbar_expect_tx(b_k_full + 8 * buf, KV_BYTES);
        for (int s = 0; s < SUB; ++s) tma_load_2d(sk + buf * KV_BYTES + s * KBOX, &map_k, kx + s * 64, row, b_k_full + 8 * buf);
        if (j >= 2) {
          ok = mbar_wait(b_v_empty + 8 * buf, ph ^ 1u, cta_abort, p.err);
          if (!ok) break;
        }
        mbar_expect_tx(b_v_full + 8 * buf, KV_BYTES);
        for (int s = 0; s < SUB; ++s) tma_load_2d(sv + buf * KV_BYTES + s * KBOX, &map_v, kx + s * 64, row, b_v_full + 8 * buf);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc(FA_BK);              // 128 x FA_BK, both operands k-major
      constexpr uint32_t idesc_o = umma_idesc(D) | (1u << 16);     // 128 x D, B operand MN-major
      bool ok = mbar_wait(b_q_full, 0, cta_abort, p.err);
      // S_j = Q K_j^T into score buffer j & 1
      auto issue_qk = [&](int j) {
        const uint32_t buf = (uint32_t)j & 1u, ph = ((uint32_t)j >> 1) & 1u;
        if (!mbar_wait(b_k_full + 8 * buf, ph, cta_abort, p.err)) return false;
        if (j >= 2 && !mbar_wait(b_s_empty + 8 * buf, ph ^ 1u, cta_abort, p.err)) return false;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
        for (int kk = 0; kk < D / UMMA_K; ++kk) {
          const uint32_t offq = (uint32_t)(kk / 4) * BOX + (uint32_t)(kk % 4) * 32u;
          const uint32_t offk = (uint32_t)(kk / 4) * KBOX + (uint32_t)(kk % 4) * 32u;
          umma_bf16(tmem_base + buf * S_COLS, umma_desc(sq + offq), umma_desc(sk + buf * KV_BYTES + offk), idesc_s,
                    kk > 0 ? 1u : 0u);
        }
        umma_commit(b_s_full + 8 * buf);
        umma_commit(b_k_empty + 8 * buf);
        return true;
      };
      // O_t = P_j V_j
      auto issue_pv = [&](int j) {
        const uint32_t buf = (uint32_t)j & 1u, ph = ((uint32_t)j >> 1) & 1u;
        if (!mbar_wait(b_p_full, (uint32_t)j & 1u, cta_abort, p.err)) return false;
        if (!mbar_wait(b_v_full + 8 * buf, ph, cta_abort, p.err)) return false;
        if (j >= 1 && !mbar_wait(b_o_empty, ((uint32_t)j & 1u) ^ 1u, cta_abort, p.err)) return false;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
#pragma unroll
        for (int kk = 0; kk < FA_BK / UMMA_K; ++kk) {
          const uint64_t da = umma_desc(sp + (uint32_t)(kk / 4) * BOX + (uint32_t)(kk % 4) * 32u);
          const uint64_t db = umma_desc_mn(sv + buf * KV_BYTES + (uint32_t)kk * (UMMA_K * 128u), KBOX);
          umma_bf16(tmem_base + O_COL, da, db, idesc_o, kk > 0 ? 1u : 0u);
        }
        umma_commit(b_o_full);
        umma_commit(b_v_empty + 8 * buf);
        umma_commit(b_p_empty);
        return true;
      };
      if (ok) ok = issue_qk(0);
      for (int j = 0; j < nt && ok; ++j) {
        if (j + 1 < nt) ok = issue_qk(j + 1);
        if (ok) ok = issue_pv(j);
      }
    }
  } else {
    const int q = warp & 3;
    const int r = q * 32 + lane;  // query row of this thread = TMEM lane
    const uint32_t lane_base = tmem_base + ((uint32_t)(q * 32) << 16);
    const int64_t qi = q0 + r;
    const int64_t qpos = start_pos + qi;
    // a gate per value: on its way into L2 long before the epilogue
    const float* wide = EXTRA && p.gate && p.wide_gate && qi < len ? p.gate + (tok0 + qi) * p.ld_gate + h * D : nullptr;
    if (wide)
#pragma unroll
      for (int i = 0; i < D; i += 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(wide + i));
    float o[D];
#pragma unroll
    for (int i = 0; i < D; ++i) o[i] = 0.f;
    float m = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = 0; j < nt && ok; ++j) {
      const uint32_t buf = (uint32_t)j & 1u, ph = ((uint32_t)j >> 1) & 1u;
      ok = mbar_wait(b_s_full + 8 * buf, ph, cta_abort, p.err);
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const int k0 = tile_of(j) * FA_BK;
      const float* bias_row = nullptr;  // of this row against the tile's keys
      if (EXTRA) {
        float* tab = bias_tab + (j & 1) * 4 * BIAS_LD;
        const float* src = p.bias + h * p.ld_bias + (start_pos + q0 - k0) + 127;
        for (int x = q * 32 + lane; x < BIAS_N; x += 128) {
          const float v = p.bias ? -LOG2E * __ldg(src - x) : 0.f;
#pragma unroll
          for (int s = 0; s < 4; ++s)
            if (x >= s) tab[s * BIAS_LD + x - s] = v;
        }
        // (a buffer is written again two tiles later, when every row has passed the barrier between)
        asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(b_bias) : "memory");
        ok = mbar_wait(b_bias, (uint32_t)j & 1u, cta_abort, p.err);
        if (!ok) break;
        bias_row = tab + ((127 - r) & 3) * BIAS_LD + ((127 - r) & ~3);
      }
      // a key column c of this tile is visible to this row iff low <= c <= lim (window and causal mask)
      // or c <= lim and c < kept; a bit per column and group of 32
      const int64_t lim64 = qpos - k0;
      const int lim = lim64 > FA_BK ? FA_BK : (lim64 < -1 ? -1 : (int)lim64);
      const int64_t low64 = p.window > 0 ? lim64 - p.window + 1 : 0;
      const int low = low64 < 0 ? 0 : (low64 > FA_BK ? FA_BK : (int)low64);
      const int64_t kept64 = p.keep - k0;
      const int kept = kept64 < 0 ? 0 : (kept64 > FA_BK ? FA_BK : (int)kept64);
      auto visible = [&](int c) {
        return bits_below(lim + 1 - c * 32) & (~bits_below(low - c * 32) | bits_below(kept - c * 32));
      };
      // uniform: some key may be masked for some row
      const bool diag = (int64_t)k0 + FA_BK - 1 > start_pos + q0 || (p.window > 0 && k0 <= last_q - p.window && kept < FA_BK);
      const uint32_t s_addr = lane_base + buf * S_COLS;
      constexpr int NCH = FA_BK / 32;
      uint32_t va[32], vb[32];
      // pass 1: row maximum of the visible scores.  The loads are double-buffered: chunk c+1 is
      // in flight while chunk c is reduced.
      float mx = -INFINITY;
      tmem_ld32(s_addr, va);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int c = 0; c < NCH; ++c) {
        uint32_t* cur = (c & 1) ? vb : va;
        uint32_t* nxt = (c & 1) ? va : vb;
        if (c + 1 < NCH) tmem_ld32(s_addr + (uint32_t)(c + 1) * 32u, nxt);
        if (!diag) {
#pragma unroll
          for (int i = 0; i < 32; ++i) mx = fmaxf(mx, __uint_as_float(cur[i]));
        } else {
          const uint32_t vis = visible(c);
#pragma unroll
          for (int i = 0; i < 32; ++i) mx = vis & (1u << i) ? fmaxf(mx, __uint_as_float(cur[i])) : mx;
        }
        if (c + 1 < NCH) asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      }
      if (EXTRA) mx = lim < 0 ? -INFINITY : mx * p.scale_log2e + fmaxf(bias_row[0], bias_row[lim < FA_BK ? lim : FA_BK - 1]);
      const float m_new = fmaxf(m, mx);
      const float m_safe = m_new == -INFINITY ? 0.f : m_new;
      const float m_unit = EXTRA ? 1.f : p.scale_log2e;             // (with EXTRA the maxima are scaled already)
      const float corr = fast_exp2((m - m_safe) * m_unit);         // 0 while m is -inf
      const float mc = m_safe * m_unit;
      // the previous tile's P must have been consumed before it is overwritten
      if (j >= 1) {
        ok = mbar_wait(b_p_empty, ((uint32_t)j & 1u) ^ 1u, cta_abort, p.err);
        if (!ok) break;
      }
      // pass 2: p = exp2(s * scale * log2 e - m * scale * log2 e), row sum, bf16 P into the swizzled tile
      float ls = 0.f;
      tmem_ld32(s_addr, va);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int c = 0; c < NCH; ++c) {
        uint32_t* cur = (c & 1) ? vb : va;
        uint32_t* nxt = (c & 1) ? va : vb;
        if (c + 1 < NCH) tmem_ld32(s_addr + (uint32_t)(c + 1) * 32u, nxt);
        const uint32_t vis = visible(c);
        uint32_t pk[16];
        float4 four = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          float t0 = -mc, t1 = -mc;
          if (EXTRA) {
            if ((i & 3) == 0) four = *(const float4*)(bias_row + c * 32 + i);
            t0 += i & 2 ? four.z : four.x;
            t1 += i & 2 ? four.w : four.y;
          }
          float e0 = fast_exp2(fmaf(__uint_as_float(cur[i]), p.scale_log2e, t0));
          float e1 = fast_exp2(fmaf(__uint_as_float(cur[i + 1]), p.scale_log2e, t1));
          if (diag) {
            e0 = vis & (1u << i) ? e0 : 0.f;
            e1 = vis & (2u << i) ? e1 : 0.f;
          }
          ls += e0 + e1;
          const __nv_bfloat162 pr = __floats2bfloat162_rn(e0, e1);
          pk[i / 2] = *(const uint32_t*)&pr;
        }
        // four 16-byte chunks of row r: chunk index ch = 4 c + t; sub-tile ch / 8, position (ch % 8) ^ (r % 8)
#pragma unroll
        for (int t = 0; t < 4; ++t) {
          const int ch = 4 * c + t;
          const uint32_t a = sp + (uint32_t)(ch / 8) * BOX + (uint32_t)r * 128u + (uint32_t)(((ch % 8) ^ (r & 7)) * 16);
          asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(a), "r"(pk[4 * t]), "r"(pk[4 * t + 1]), "r"(pk[4 * t + 2]),
                       "r"(pk[4 * t + 3])
                       : "memory");
        }
        if (c + 1 < NCH) asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      }
      // S buffer free for the tile after next; P visible to the tensor core
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(b_s_empty + 8 * buf) : "memory");
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(b_p_full) : "memory");
      l = l * corr + ls;
      m = m_new;
      // fold O_t = P V into the running output (same double-buffered loads)
      ok = mbar_wait(b_o_full, (uint32_t)j & 1u, cta_abort, p.err);
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      tmem_ld32(lane_base + O_COL, va);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int c = 0; c < D / 32; ++c) {
        uint32_t* cur = (c & 1) ? vb : va;
        uint32_t* nxt = (c & 1) ? va : vb;
        if (c + 1 < D / 32) tmem_ld32(lane_base + O_COL + (uint32_t)(c + 1) * 32u, nxt);
#pragma unroll
        for (int i = 0; i < 32; ++i) o[c * 32 + i] = fmaf(o[c * 32 + i], corr, __uint_as_float(cur[i]));
        if (c + 1 < D / 32) asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      }
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(b_o_empty) : "memory");
    }
    if (ok && qi < len) {
      float inv = l > 0.f ? 1.f / l : 0.f;
      if (p.sink) {
        // one more term of the denominator, without a value
        const float mc = EXTRA ? m : m * p.scale_log2e, sk = p.sink[h] * LOG2E, top = fmaxf(mc, sk);
        const float f = fast_exp2(mc - top);
        inv = f / (l * f + fast_exp2(sk - top));
      }
      inv *= p.out_scale;
      if (p.gate && !p.wide_gate) inv *= 1.f / (1.f + expf(-p.gate[(tok0 + qi) * p.ld_gate + h]));
      if (EXTRA && wide) {
        // 64 gates at a time, all requested before the first is used
#pragma unroll
        for (int c0 = 0; c0 < D; c0 += 64) {
          float4 g[16];
#pragma unroll
          for (int i = 0; i < 16; ++i) g[i] = __ldg((const float4*)(wide + c0) + i);
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            float* x = o + c0 + 4 * i;
            x[0] *= sigmoid_fast(g[i].x); x[1] *= sigmoid_fast(g[i].y); x[2] *= sigmoid_fast(g[i].z); x[3] *= sigmoid_fast(g[i].w);
          }
        }
      }
      __nv_bfloat16* dst = p.out + (tok0 + qi) * p.ld_out + (int64_t)h * D;
#pragma unroll
      for (int c0 = 0; c0 < D; c0 += 8) {
        uint32_t w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const __nv_bfloat162 pr = __floats2bfloat162_rn(o[c0 + 2 * i] * inv, o[c0 + 2 * i + 1] * inv);
          w[i] = *(const uint32_t*)&pr;
        }
        *(uint4*)(dst + c0) = make_uint4(w[0], w[1], w[2], w[3]);
      }
    }
  }

  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    __syncwarp();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(NCOLS) : "memory");
  }
}

template <int D, int FA_BK, bool EXTRA>
int launch_fa(cg_ctx* c, const AttnArgs& a) {
  constexpr size_t smem =
      (size_t)(D / 64) * (128 + 4 * FA_BK) * 128 + (size_t)(FA_BK / 64) * 128 * 128 + (FA_BK == 64 ? 0 : 1024) + 160 +
      (EXTRA ? (size_t)2 * 4 * (127 + FA_BK + 9) * 4 : 0);
  static PerDeviceFlag configured_on;
  bool& configured = configured_on.at(c->core->device);
  if (!configured) {
    CG_CUDA(c, cudaFuncSetAttribute(k_attn_fa<D, FA_BK, EXTRA>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    configured = true;
  }
  CUtensorMap mq, mk, mv;
  CG_TRY(make_map(c, &mq, a.q, a.rows.rows ? a.rows.M : a.B * a.S, (int64_t)a.nh * D, (int64_t)a.nh * D, 128));
  const bool tm = a.kv_ld > 0;
  const int64_t kv_rows = tm ? a.B * a.Tmax : a.B * a.nkv * a.Tmax, kv_cols = tm ? (int64_t)a.nkv * D : D, kv_ld = tm ? a.kv_ld : D;
  CG_TRY(make_map(c, &mk, a.k_cache, kv_rows, kv_cols, kv_ld, FA_BK));
  CG_TRY(make_map(c, &mv, a.v_cache, kv_rows, kv_cols, kv_ld, FA_BK));
  FaArgs p;
  p.out = a.out;
  p.S = a.S; p.pos0 = a.pos0; p.Tmax = a.Tmax;
  p.nh = a.nh; p.nkv = a.nkv;
  p.token_major = tm ? 1 : 0;
  p.scale_log2e = 1.4426950408889634f * (a.scale > 0.f ? a.scale : 1.f / sqrtf((float)D));
  p.window = a.window > 0 ? a.window : 0;
  p.keep = p.window ? std::max<int64_t>(a.keep_first, 0) : 0;
  p.sink = a.sink;
  p.wide_gate = a.wide_gate; p.bias = a.bias; p.ld_bias = a.ld_bias;
  p.gate = a.gate; p.ld_gate = a.ld_gate; p.out_scale = a.out_scale;
  p.ld_out = a.ld_out > 0 ? a.ld_out : (int64_t)a.nh * D;
  p.rows = a.rows;
  p.err = c->core->dev_err;
  dim3 grid((unsigned)((a.S + FA_BQ - 1) / FA_BQ), (unsigned)a.nh, (unsigned)(a.rows.rows ? a.rows.rows : a.B));
  CG_CUDA(c, launch_kernel(c, k_attn_fa<D, FA_BK, EXTRA>, grid, dim3(192), smem, 1, mq, mk, mv, p));
  CG_LAUNCHED(c);
  return CG_OK;
}

}  // namespace

bool attn_fa_supported(const AttnArgs& a) {
  return (a.d == 64 || a.d == 128) && a.softcap <= 0.f && !a.pos_dev && a.S >= 64 &&
         (a.rows.rows ? a.rows.M : a.B * a.S) < 2147483647ll && a.B * a.nkv * a.Tmax < 2147483647ll && ((uintptr_t)a.q % 16) == 0 &&
         ((uintptr_t)a.k_cache % 16) == 0 && ((uintptr_t)a.v_cache % 16) == 0 && a.kv_ld % 8 == 0 && ((uintptr_t)a.out % 16) == 0 && a.ld_out % 8 == 0 &&
         (!a.wide_gate || (((uintptr_t)a.gate % 16) == 0 && a.ld_gate % 4 == 0));
}

int k_launch_attn_fa(cg_ctx* c, const AttnArgs& a) {
  if (a.B == 0 || a.S == 0) return CG_OK;
  // 64-key tiles: two CTAs per SM.  Head size 64 gains from it (8 x 1024 tokens, 64 heads: 380 -> 315 us,
  // with a window of 128 225 -> 165 us), head size 128 does not (242 -> 264 us).
  const bool k64 = c->opt_fa == 2 || a.d == 64;
  if (a.bias || (a.gate && a.wide_gate)) {
    if (a.d == 64) return launch_fa<64, 64, true>(c, a);
    return k64 ? launch_fa<128, 64, true>(c, a) : launch_fa<128, 128, true>(c, a);
  }
  if (a.d == 64) return k64 ? launch_fa<64, 64, false>(c, a) : launch_fa<64, 128, false>(c, a);
  return k64 ? launch_fa<128, 64, false>(c, a) : launch_fa<128, 128, false>(c, a);
}

}  // namespace cg
