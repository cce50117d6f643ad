// Prefill attention with an optional sliding window (which may keep the first tokens of the sequence) or chunk mask, soft-capped scores,
// a sink per head in the softmax or sigmoid weights in its place, and outputs turned back by the query's position, for sm_100a
// (tcgen05 + TMEM).
//
// Keys and values are contiguous rows (the expanded latents of the keys a batch reads, one head per query head) or the cache pages
// themselves (grouped-query attention: a step of 64 keys lies inside one 128-token page).  One CTA owns one head and up to 256
// consecutive new tokens of one request as two blocks of 128 query rows; both blocks read the same 64-key K / V steps, loaded once,
// and their softmax runs on two warp groups, so the tensor core alternates between the blocks:
//     S_b[128 q x 64 k] = Q_b * K^T        O_b[128 q x V] += P_b * V          b = 0, 1
// A block takes part only in the steps its rows see (the causal frontier at one end, the window at the other).  Head widths are
// any multiple of 8: the operand maps are bounded per head, so the tail of a 64-column tile is zero.  Kept first tokens are steps of
// their own ahead of the window's, shared by both blocks.  Expanded keys may be followed by a part that all heads share (rotated
// dimensions): its tiles come from the shared rows, the queries' from behind every head's own dimensions.  The epilogue normalises (with the sink's term) and applies the output gate
// o * sigmoid(g), one per element or one per head, where the layer has one.
#include "ptx.cuh"
#include "launch.h"
#include "tmap.h"

FB_DEFINE_ERROR_API(attn_window)

namespace fb {

constexpr int KID_ATTN_WINDOW = 16;
constexpr int AW_KV = 64;                          // keys per step
constexpr int AW_QT = 128 * 128;                   // bytes of a [128 rows x 64 cols] tile
constexpr int AW_KT = AW_KV * 128;                 // bytes of a [64 rows x 64 cols] tile
constexpr int AW_PT = 128 * AW_KV * 2;
constexpr int AW_SMEM_MAX = 227 * 1024;

struct AttnWindowParams {
  // [n_blocks][6] = packed row of the first query, its position, query rows (<= 256), row of the request's first key, that key's
  // position, request (row of the page table)
  const int* blocks;
  uint16_t* out; long long ld_out;
  const uint16_t* gate; long long ld_gate;
  int D, V, dt, vt;                               // head widths, their 64-column tiles
  int R, rt;                                      // width of the shared key part (0: none) and its tiles, behind the dt tiles of D
  int stages, window;
  int chunk;                                      // > 0 (instead of a window): a query sees the keys of its own chunk of positions
  int group;                                      // query heads per key / value head
  const int* page_table; int max_pages, num_pages;     // null: contiguous keys
  int keep;                                       // pages only, beside a window: the first `keep` keys stay visible
  float scale_log2;
  float cap_log2, cap_in;                         // soft cap c: c log2(e), 2 log2(e) scale / c (0: none)
  float cap_lim, cap_p[6];                        // products up to cap_lim: the capped score is s * polynomial(s^2)
  const float* sinks;                             // [heads] or null
  const float* head_gate; long long ld_head_gate;      // one logit per (row, head)
  const float* score_bias;                        // [heads]: the weight of a key is sigmoid(score + score_bias[h]) (null: softmax)
  const float* cos_v; const float* sin_v;         // [tab_rows, rot_v / 2]: output pairs (2m, 2m + 1) are turned back by the position
  int rot_v, tab_rows;
  uint32_t idesc_s, idesc_o;
};

// first position a query at `pos` sees
__device__ __forceinline__ int aw_first(const AttnWindowParams& p, int pos) {
  if (p.chunk > 0) return pos - pos % p.chunk;
  return p.window > 0 ? pos - p.window + 1 : 0;
}

// tanh(x) / x on |x| <= AW_TANH_LIM as a polynomial in x^2: least squares on Chebyshev nodes, reweighted until the error is level
// (|error of tanh| <= 2e-8)
constexpr float AW_TANH_LIM = 0.8f;
constexpr float AW_TANH[6] = {0.99999967f, -0.33331833f, 0.1331374f, -0.05285472f, 0.01868937f, -0.00412656f};

// c tanh(x): 1 - 2 / (1 + e^2x) is exact to an fp32 rounding of one, which is all that a score needs
__device__ __forceinline__ float aw_capped(const AttnWindowParams& p, float s) {
  return p.cap_log2 - __fdividef(2.f * p.cap_log2, 1.f + exp2f(s * p.cap_in));
}

// MODE: 0 plain softmax; 1 soft cap, kept tokens, sinks, head gates and turned outputs are looked at; 2 sigmoid weights, with all of these
// but sinks
template <bool BF16, int MODE>
__global__ void __launch_bounds__(320, 1)
attn_window_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                   const __grid_constant__ CUtensorMap tmQr, const __grid_constant__ CUtensorMap tmKr, const AttnWindowParams p) {
  constexpr bool EXT = MODE != 0;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int own = p.dt, dt = own + p.rt, vt = p.vt, stages = p.stages;
  const int stage_bytes = (dt + vt) * AW_KT;
  uint8_t* q_smem = smem;                                   // [2 blocks][dt] tiles of 16 KB
  uint8_t* kv_smem = smem + 2 * dt * AW_QT;                 // [stages] x (K tiles, V tiles)
  uint8_t* p_smem = kv_smem + stages * stage_bytes;         // [2 blocks] x 16 KB
  uint64_t* bars = reinterpret_cast<uint64_t*>(p_smem + 2 * AW_PT);
  uint64_t* full_k = bars;                                  // [4]
  uint64_t* full_v = bars + 4;
  uint64_t* empty = bars + 8;
  uint64_t* q_full = bars + 12;
  uint64_t* s_full = bars + 13;       // [2]
  uint64_t* p_ready = bars + 15;      // [2]
  uint64_t* o_full = bars + 17;       // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 19);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.x, kv_head = head / p.group;
  const int* blk = p.blocks + 6 * blockIdx.y;
  const int q_row0 = blk[0], pos0 = blk[1], rows = blk[2], key_row0 = blk[3], key0 = blk[4];
  // first key of the block's first row, one past the last key of its last row
  int lo = max(key0, aw_first(p, pos0));
  if (p.page_table != nullptr) lo &= ~(AW_KV - 1);          // a step never straddles two pages; the mask drops what lies before
  const int hi = pos0 + rows;
  const int kept = EXT && p.keep > 0 ? min((p.keep + AW_KV - 1) / AW_KV, lo / AW_KV) : 0;      // steps of kept tokens before the window's
  const int n_steps = kept + (hi - lo + AW_KV - 1) / AW_KV;
  auto step_key = [&](int it) { return EXT && it < kept ? it * AW_KV : lo + (it - kept) * AW_KV; };
  // query block b takes part in steps [0, kb) and [f, e); its n-th step is nth(b, n)
  int f[2], e[2], kb[2];
  kb[0] = f[0] = kept;
  e[0] = kept + (pos0 + (rows < 128 ? rows : 128) - lo + AW_KV - 1) / AW_KV;
  if (rows > 128) {
    kb[1] = kept;
    f[1] = kept + (EXT && p.keep > lo ? 0 : (max(lo, aw_first(p, pos0 + 128)) - lo) / AW_KV);
    e[1] = n_steps;
  } else {
    kb[1] = 0;
    f[1] = e[1] = n_steps;
  }
  auto takes = [&](int b, int it) { return (EXT && it < kb[b]) || (it >= f[b] && it < e[b]); };
  auto order = [&](int b, int it) { return EXT ? (it < kb[b] ? it : kb[b] + it - f[b]) : it - f[b]; };
  bool dead = false;

  if (threadIdx.x == 0) {
    for (int s = 0; s < stages; ++s) { mbar_init(&full_k[s], 1); mbar_init(&full_v[s], 1); mbar_init(&empty[s], 1); }
    mbar_init(q_full, 1);
    for (int b = 0; b < 2; ++b) { mbar_init(&s_full[b], 1); mbar_init(&p_ready[b], 128); mbar_init(&o_full[b], 1); }
    mbar_init_fence();
    tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, 512); tmem_relinquish(); }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem0 = *tmem_slot;
  // columns: S_0 [0,64) S_1 [64,128) O_0 [128, 128 + 64 vt) O_1 behind it
  const uint32_t o_cols = (uint32_t)(vt * 64);

  if (warp == 0) {
    if (elect_one()) {
      const int nb = rows > 128 ? 2 : 1;
      mbar_expect_tx(q_full, nb * dt * AW_QT);
      for (int b = 0; b < nb; ++b)
        for (int j = 0; j < dt; ++j)
          tma_load_3d(q_smem + (b * dt + j) * AW_QT, j < own ? &tmQ : &tmQr, q_full, (j < own ? j : j - own) * 64, head, q_row0 + b * 128);
      for (int it = 0; it < n_steps; ++it) {
        const int s = it % stages;
        const uint32_t ph = (uint32_t)(it / stages) & 1u;
        if (!mbar_wait(&empty[s], ph ^ 1u, dead, KID_ATTN_WINDOW, 1)) break;
        const int key = step_key(it);
        int row = key_row0 + (key - key0);
        if (p.page_table != nullptr) {
          int page = (key >> 7) < p.max_pages ? p.page_table[(size_t)blk[5] * p.max_pages + (key >> 7)] : 0;
          if ((unsigned)page >= (unsigned)p.num_pages) { report_error(ERR_BAD_ARG, KID_ATTN_WINDOW, 20); page = 0; }
          row = page * 128 + (key & 127);
        }
        uint8_t* ks = kv_smem + s * stage_bytes;
        uint8_t* vb = ks + dt * AW_KT;
        mbar_expect_tx(&full_k[s], dt * AW_KT);
        for (int j = 0; j < own; ++j) tma_load_3d(ks + j * AW_KT, &tmK, &full_k[s], j * 64, kv_head, row);
        for (int j = own; j < dt; ++j) tma_load_3d(ks + j * AW_KT, &tmKr, &full_k[s], (j - own) * 64, 0, row);
        mbar_expect_tx(&full_v[s], vt * AW_KT);
        for (int j = 0; j < vt; ++j) tma_load_3d(vb + j * AW_KT, &tmV, &full_v[s], j * 64, kv_head, row);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (elect_one()) {
      const uint32_t qb = smem_u32(q_smem), pb = smem_u32(p_smem);
      const int ks = (p.D + 15) / 16, kr = 4 * own, kre = kr + (p.R + 15) / 16;       // 16-wide k steps of the S product: [0, ks) and [kr, kre)
      auto issue_s = [&](int b, uint32_t kb) {
        for (int k = 0; k < kre; k = k + 1 == ks ? kr : k + 1) {
          const uint64_t da = make_smem_desc(qb + (b * dt + (k >> 2)) * AW_QT + (k & 3) * 32, 16, 1024, SWZ_128B);
          const uint64_t db = make_smem_desc(kb + (k >> 2) * AW_KT + (k & 3) * 32, 16, 1024, SWZ_128B);
          umma_f16(tmem0 + (uint32_t)(b * 64), da, db, p.idesc_s, k != 0 ? 1u : 0u);
        }
        umma_commit(&s_full[b]);
      };
      bool ok = mbar_wait(q_full, 0, dead, KID_ATTN_WINDOW, 2);
      if (ok) ok = mbar_wait(&full_k[0], 0, dead, KID_ATTN_WINDOW, 3);
      if (ok) {
        tc_fence_after_sync();
        for (int b = 0; b < 2; ++b)
          if (takes(b, 0)) issue_s(b, smem_u32(kv_smem));
      }
      for (int it = 0; ok && it < n_steps; ++it) {
        const int s = it % stages, s1 = (it + 1) % stages;
        const uint32_t ph = (uint32_t)(it / stages) & 1u, ph1 = (uint32_t)((it + 1) / stages) & 1u;
        const uint32_t vb = smem_u32(kv_smem + s * stage_bytes + dt * AW_KT);
        const uint32_t kb1 = smem_u32(kv_smem + s1 * stage_bytes);
        bool have_v = false, have_k1 = false;
        for (int b = 0; b < 2; ++b) {
          if (takes(b, it)) {
            if (!mbar_wait(&p_ready[b], (uint32_t)order(b, it) & 1u, dead, KID_ATTN_WINDOW, 4)) { ok = false; break; }
            if (!have_v && !mbar_wait(&full_v[s], ph, dead, KID_ATTN_WINDOW, 5)) { ok = false; break; }
            have_v = true;
            tc_fence_after_sync();
            // O_b += P_b * V : A = P_b (K-major, 64 keys), B = V step MN-major (16 keys per MMA)
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              const uint64_t da = make_smem_desc(pb + b * AW_PT + k * 32, 16, 1024, SWZ_128B);
              const uint64_t db = make_smem_desc(vb + k * 2048, AW_KT, 1024, SWZ_128B);
              umma_f16(tmem0 + 128u + (uint32_t)b * o_cols, da, db, p.idesc_o, (order(b, it) != 0 || k != 0) ? 1u : 0u);
            }
            umma_commit(&o_full[b]);
          }
          if (takes(b, it + 1)) {
            if (!have_k1 && !mbar_wait(&full_k[s1], ph1, dead, KID_ATTN_WINDOW, 6)) { ok = false; break; }
            have_k1 = true;
            tc_fence_after_sync();
            issue_s(b, kb1);
          }
        }
        if (ok) {
          // (a step no block used for V has its load outstanding: the slot may only be refilled once it has landed)
          if (!have_v && !mbar_wait(&full_v[s], ph, dead, KID_ATTN_WINDOW, 7)) break;
          umma_commit(&empty[s]);
        }
      }
    }
    __syncwarp();
  } else {
    const int b = (warp - 2) >> 2;               // query block of this warp group
    const int q = warp & 3;                      // TMEM lane quarter: warps 2..5 -> 2,3,0,1 ; 6..9 -> 2,3,0,1
    const int r = q * 32 + lane;
    const int pos_b = pos0 + b * 128, pos = pos_b + r;
    const int first = aw_first(p, pos), first_all = aw_first(p, pos_b + 127);      // of this row; no earlier than any row of the block's
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    const uint32_t tmem_s = tmem0 + (uint32_t)(b * 64), tmem_o = tmem0 + 128u + (uint32_t)b * o_cols;
    uint8_t* prow = p_smem + b * AW_PT + r * 128;
    const int cnt = (EXT ? kb[b] : 0) + e[b] - f[b];
    float m_run = -INFINITY, l_run = 0.f;
    const float bias = MODE == 2 ? p.score_bias[head] * 1.4426950408889634f : 0.f;
    for (int n = 0; n < cnt; ++n) {
      const uint32_t iph = (uint32_t)n & 1u;
      mbar_wait(&s_full[b], iph, dead, KID_ATTN_WINDOW, 8);
      tc_fence_after_sync();
      const int kv0 = EXT ? step_key(n < kb[b] ? n : f[b] + n - kb[b]) : lo + (f[b] + n) * AW_KV;
      uint32_t sreg[64];
      tmem_ld_32x32b_x32(tmem_s + lane_off, sreg);
      tmem_ld_32x32b_x32(tmem_s + lane_off + 32, sreg + 32);
      tmem_ld_wait();
      // only steps on the causal diagonal or on the window's edge pay for the mask
      const bool full_step = kv0 + AW_KV - 1 <= pos_b && (kv0 >= first_all || (EXT && kv0 + AW_KV <= p.keep));
      float m_new = m_run;
      const bool cap = EXT && p.cap_in != 0.f;
      if (cap) {
        float am = 0.f;
#pragma unroll
        for (int j = 0; j < 64; ++j) am = fmaxf(am, fabsf(__uint_as_float(sreg[j])));
        if (__all_sync(0xffffffffu, am <= p.cap_lim)) {
          uint64_t cf[6];
#pragma unroll
          for (int i = 0; i < 6; ++i) cf[i] = pack_f32x2(p.cap_p[i], p.cap_p[i]);
#pragma unroll
          for (int j = 0; j < 64; j += 2) {
            const uint64_t s = pack_f32x2(__uint_as_float(sreg[j]), __uint_as_float(sreg[j + 1])), u = mul_f32x2(s, s);
            uint64_t y = cf[5];
#pragma unroll
            for (int i = 4; i >= 0; --i) y = fma_f32x2(u, y, cf[i]);
            float a, c;
            unpack_f32x2(mul_f32x2(s, y), a, c);
            sreg[j] = __float_as_uint(a);
            sreg[j + 1] = __float_as_uint(c);
          }
        } else {
#pragma unroll
          for (int j = 0; j < 64; ++j) sreg[j] = __float_as_uint(aw_capped(p, __uint_as_float(sreg[j])));
        }
      }
      const float sc = cap ? 1.f : p.scale_log2;
      if (MODE == 2) {
        // P = sigmoid(score + bias): no maximum, no sum, nothing to rescale; one reciprocal serves two scores (clamped so that the
        // product of two denominators stays finite: a weight below 2^-60 counts as that)
        if (n > 0) {
          mbar_wait(&o_full[b], iph ^ 1u, dead, KID_ATTN_WINDOW, 9);
          tc_fence_after_sync();
        }
#pragma unroll
        for (int g = 0; g < 8; ++g) {
          uint32_t pk[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const int c = 8 * g + 2 * j, kv = kv0 + c;
            const float a0 = 1.f + exp2f(fminf(-fmaf(__uint_as_float(sreg[c]), sc, bias), 60.f));
            const float a1 = 1.f + exp2f(fminf(-fmaf(__uint_as_float(sreg[c + 1]), sc, bias), 60.f));
            const float inv = __fdividef(1.f, a0 * a1);
            float p0 = inv * a1, p1 = inv * a0;
            if (!full_step) {
              if (!(kv <= pos && (kv >= first || kv < p.keep))) p0 = 0.f;
              if (!(kv + 1 <= pos && (kv + 1 >= first || kv + 1 < p.keep))) p1 = 0.f;
            }
            pk[j] = pack_16<BF16>(p0, p1);
          }
          *reinterpret_cast<uint4*>(prow + ((g ^ (r & 7)) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
        }
        fence_proxy_async_smem();
        tc_fence_before_sync();
        mbar_arrive(&p_ready[b]);
        continue;
      }
      if (full_step) {
#pragma unroll
        for (int j = 0; j < 64; ++j) {
          const float sv = __uint_as_float(sreg[j]) * sc;
          sreg[j] = __float_as_uint(sv);
          m_new = fmaxf(m_new, sv);
        }
      } else {
#pragma unroll
        for (int j = 0; j < 64; ++j) {
          const int kv = kv0 + j;
          const float sv = (kv <= pos && (kv >= first || (EXT && kv < p.keep))) ? __uint_as_float(sreg[j]) * sc : -INFINITY;
          sreg[j] = __float_as_uint(sv);
          m_new = fmaxf(m_new, sv);
        }
      }
      const float m_use = m_new == -INFINITY ? 0.f : m_new;
      const float alpha = exp2f(m_run - m_use);
      if (n > 0) {
        // the previous P * V of this block must be complete before P is overwritten or O is rescaled
        mbar_wait(&o_full[b], iph ^ 1u, dead, KID_ATTN_WINDOW, 9);
        tc_fence_after_sync();
        if (__any_sync(0xffffffffu, alpha != 1.0f)) {
#pragma unroll 1
          for (int c0 = 0; c0 < (int)o_cols; c0 += 32) {
            uint32_t oreg[32];
            tmem_ld_32x32b_x32(tmem_o + lane_off + c0, oreg);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 32; ++j) oreg[j] = __float_as_uint(__uint_as_float(oreg[j]) * alpha);
            tmem_st_32x32b_x32(tmem_o + lane_off + c0, oreg);
          }
          tmem_st_wait();
        }
      }
      float l_add = 0.f;
#pragma unroll
      for (int g = 0; g < 8; ++g) {
        uint32_t pk[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float p0 = exp2f(__uint_as_float(sreg[8 * g + 2 * j]) - m_use);
          const float p1 = exp2f(__uint_as_float(sreg[8 * g + 2 * j + 1]) - m_use);
          pk[j] = pack_16<BF16>(p0, p1);
          l_add += p0 + p1;
        }
        *reinterpret_cast<uint4*>(prow + ((g ^ (r & 7)) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
      }
      l_run = l_run * alpha + l_add;
      m_run = m_new;
      fence_proxy_async_smem();
      tc_fence_before_sync();
      mbar_arrive(&p_ready[b]);
    }
    if (cnt > 0) {
      mbar_wait(&o_full[b], (uint32_t)(cnt - 1) & 1u, dead, KID_ATTN_WINDOW, 10);
      tc_fence_after_sync();
      float inv_l = MODE == 2 ? 1.f : l_run > 0.f ? 1.f / l_run : 0.f;
      const bool live = b * 128 + r < rows;
      const size_t row = (size_t)(q_row0 + b * 128 + r);
      if (MODE == 1 && p.sinks != nullptr && l_run > 0.f) {
        const float sink = p.sinks[head] * 1.4426950408889634f, mx = fmaxf(m_run, sink), fac = exp2f(m_run - mx);
        inv_l = fac / (l_run * fac + exp2f(sink - mx));
      }
      if (EXT && p.head_gate != nullptr && live) inv_l *= 1.0f / (1.0f + __expf(-p.head_gate[row * p.ld_head_gate + head]));
      uint16_t* orow = p.out + row * p.ld_out + (size_t)head * p.V;
      const uint16_t* grow = p.gate != nullptr ? p.gate + row * p.ld_gate + (size_t)head * p.V : nullptr;
#pragma unroll 1
      for (int c0 = 0; c0 < p.V; c0 += 32) {
        uint32_t oreg[32];
        __syncwarp();
        tmem_ld_32x32b_x32(tmem_o + lane_off + c0, oreg);
        tmem_ld_wait();
        if (live) {
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            if (c0 + 8 * g >= p.V) break;
            float v[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) v[j] = __uint_as_float(oreg[8 * g + j]) * inv_l;
            if (EXT && p.rot_v > 0) {
              const int half = p.rot_v >> 1, m0 = (c0 + 8 * g) >> 1;
              const size_t at = (size_t)(pos < p.tab_rows ? pos : p.tab_rows - 1) * half + m0;
              float cs[4], sn[4];
              if ((half & 3) == 0 && m0 < half) {
                const float4 a = *reinterpret_cast<const float4*>(p.cos_v + at), c = *reinterpret_cast<const float4*>(p.sin_v + at);
                cs[0] = a.x; cs[1] = a.y; cs[2] = a.z; cs[3] = a.w;
                sn[0] = c.x; sn[1] = c.y; sn[2] = c.z; sn[3] = c.w;
              } else {
#pragma unroll
                for (int j = 0; j < 4; ++j) { cs[j] = m0 + j < half ? p.cos_v[at + j] : 1.f; sn[j] = m0 + j < half ? p.sin_v[at + j] : 0.f; }
              }
#pragma unroll
              for (int j = 0; j < 4; ++j) {
                const float u = v[2 * j], w = v[2 * j + 1];
                v[2 * j] = u * cs[j] + w * sn[j];
                v[2 * j + 1] = w * cs[j] - u * sn[j];
              }
            }
            if (grow != nullptr) {
              const uint4 gv = *reinterpret_cast<const uint4*>(grow + c0 + 8 * g);
              const float2 g0 = unpack_16<BF16>(gv.x), g1 = unpack_16<BF16>(gv.y), g2 = unpack_16<BF16>(gv.z), g3 = unpack_16<BF16>(gv.w);
              const float gg[8] = {g0.x, g0.y, g1.x, g1.y, g2.x, g2.y, g3.x, g3.y};
#pragma unroll
              for (int j = 0; j < 8; ++j) v[j] *= 1.0f / (1.0f + __expf(-gg[j]));
            }
            *reinterpret_cast<uint4*>(orow + c0 + 8 * g) =
                make_uint4(pack_16<BF16>(v[0], v[1]), pack_16<BF16>(v[2], v[3]), pack_16<BF16>(v[4], v[5]), pack_16<BF16>(v[6], v[7]));
          }
        }
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem0, 512);
}

// Ring depth that fits beside the queries and probabilities; 0: the head widths are outside the kernel.
static int window_stages(int D, int R, int V) {
  const int dt = (D + 63) / 64 + (R + 63) / 64, vt = (V + 63) / 64;
  if (vt > 3) return 0;                                       // 2 accumulators of 64 vt columns beside S: 512 TMEM columns
  const int fixed = 2 * dt * AW_QT + 2 * AW_PT + 256 + 1024;
  const int n = (AW_SMEM_MAX - fixed) / ((dt + vt) * AW_KT);
  return n < 2 ? 0 : n > 4 ? 4 : n;
}

}  // namespace fb

using namespace fb;

// D: a head's own key dimensions, R: those all heads share
extern "C" int fb_attn_window_supported(int D, int R, int V) {
  return D > 0 && R >= 0 && V > 0 && D % 8 == 0 && R % 8 == 0 && V % 8 == 0 && window_stages(D, R, V) > 0 ? 1 : 0;
}

static int launch_window(const CUtensorMap& tmQ, const CUtensorMap& tmK, const CUtensorMap& tmV, const CUtensorMap& tmQr, const CUtensorMap& tmKr,
                         AttnWindowParams p, int n_blocks, int H, float scale, int dtype, cudaStream_t stream) {
  p.dt = (p.D + 63) / 64; p.rt = (p.R + 63) / 64; p.vt = (p.V + 63) / 64; p.stages = window_stages(p.D, p.R, p.V);
  p.scale_log2 = scale * 1.4426950408889634f;
  const uint32_t fm = dtype == 1 ? 1u : 0u;
  p.idesc_s = make_idesc(fm, fm, 0, 0, 128, AW_KV);
  p.idesc_o = make_idesc(fm, fm, 0, 1, 128, p.vt * 64);
  const int tiles = p.dt + p.rt, smem = 2 * tiles * AW_QT + p.stages * (tiles + p.vt) * AW_KT + 2 * AW_PT + 256 + 1024;
  const dim3 grid(H, n_blocks);
#define FB_AW(BF, MODE)                                                                                                             \
  {                                                                                                                                  \
    static DeviceOnce cfg;                                                                                                           \
    if (cfg.need()) cudaFuncSetAttribute(attn_window_kernel<BF, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, AW_SMEM_MAX);      \
    attn_window_kernel<BF, MODE><<<grid, 320, smem, stream>>>(tmQ, tmK, tmV, tmQr, tmKr, p);                                         \
  }
  if (p.score_bias != nullptr) { if (dtype == 1) FB_AW(true, 2) else FB_AW(false, 2) }
  else if (p.cap_in != 0.f || p.keep > 0 || p.sinks != nullptr || p.head_gate != nullptr || p.rot_v > 0) { if (dtype == 1) FB_AW(true, 1) else FB_AW(false, 1) }
  else { if (dtype == 1) FB_AW(true, 0) else FB_AW(false, 0) }
#undef FB_AW
  return (int)cudaGetLastError();
}

// q: packed rows [T, >= H * q_head] (row stride ld_q; a head is [D own | R shared-part dimensions | padding], q_head apart), k: [n_keys, >= H * D],
// v: [n_keys, >= H * V], k_shared: [n_keys, >= R] (R = 0: none), out [T, H * V], gate (optional) like out, head_gate (optional): fp32
// logits, one per (row, head).
extern "C" int fb_attn_window(const void* q, long long ld_q, int q_head, int T, const void* k, long long ld_k, const void* v, long long ld_v, const void* k_shared,
                              long long ld_shared, int n_keys, void* out, long long ld_out, const void* gate, long long ld_gate, const float* head_gate,
                              long long ld_head_gate, const int* blocks, int n_blocks, int H, int D, int R, int V, int window, float scale, int dtype,
                              void* stream_) {
  if (n_blocks <= 0) return 0;
  if (D <= 0 || R < 0 || V <= 0 || window_stages(D, R, V) == 0 || D % 8 != 0 || R % 8 != 0 || V % 8 != 0 || q_head < D + R || q_head % 8 != 0 || T <= 0 || n_keys <= 0 || H <= 0 ||
      n_blocks > 65535 || window < 0 || ld_out % 8 != 0 || ld_gate % 8 != 0 || (R > 0 && k_shared == nullptr))
    return -1;
  CUtensorMap tmQ, tmK, tmV, tmQr, tmKr;
  if (!make_tmap_3d(&tmQ, q, D, H, T, q_head, ld_q, 64, 128)) return -2;
  if (!make_tmap_3d(&tmK, k, D, H, n_keys, D, ld_k, 64, AW_KV)) return -2;
  if (!make_tmap_3d(&tmV, v, V, H, n_keys, V, ld_v, 64, AW_KV)) return -2;
  tmQr = tmQ; tmKr = tmK;
  if (R > 0 && !make_tmap_3d(&tmQr, reinterpret_cast<const uint16_t*>(q) + D, R, H, T, q_head, ld_q, 64, 128)) return -2;
  if (R > 0 && !make_tmap_3d(&tmKr, k_shared, R, 1, n_keys, R, ld_shared, 64, AW_KV)) return -2;
  AttnWindowParams p = {};
  p.blocks = blocks; p.out = (uint16_t*)out; p.ld_out = ld_out; p.gate = (const uint16_t*)gate; p.ld_gate = ld_gate;
  p.D = D; p.R = R; p.V = V; p.window = window; p.group = 1; p.head_gate = head_gate; p.ld_head_gate = ld_head_gate;
  return launch_window(tmQ, tmK, tmV, tmQr, tmKr, p, n_blocks, H, scale, dtype, reinterpret_cast<cudaStream_t>(stream_));
}

// Grouped-query form over the cache pages: k_pool [num_slots, G, D], v_pool [num_slots, G, V], 128 slots a page; H / G
// consecutive query heads share a key / value head; keep, softcap, sinks, head_gate, score_bias and the output's rotation as in fb_grouped_decode.  page_table: [requests, max_pages], a block's request is blocks[.][5].
extern "C" int fb_attn_window_paged(const void* q, long long ld_q, int T, const void* k_pool, const void* v_pool, long long num_slots,
                                    const int* page_table, int max_pages, void* out, long long ld_out, const void* gate, long long ld_gate,
                                    const int* blocks, int n_blocks, int H, int G, int D, int V, int window, int chunk, int keep, float scale,
                                    float softcap, const float* sinks, const float* head_gate, long long ld_head_gate, const float* score_bias, const float* cos_v,
                                    const float* sin_v, int rot_v, int tab_rows, int dtype, void* stream_) {
  if (n_blocks <= 0) return 0;
  if (D <= 0 || V <= 0 || window_stages(D, 0, V) == 0 || rot_v < 0 || (rot_v & 1) || rot_v > V || (score_bias != nullptr && sinks != nullptr) ||
      (rot_v > 0 && (cos_v == nullptr || sin_v == nullptr || tab_rows <= 0)) || D % 8 != 0 || V % 8 != 0 || T <= 0 || num_slots < 128 || H <= 0 || G <= 0 || H % G != 0 || n_blocks > 65535 ||
      window < 0 || chunk < 0 || keep < 0 || softcap < 0.f || max_pages <= 0 || ld_out % 8 != 0 || ld_gate % 8 != 0)
    return -1;
  CUtensorMap tmQ, tmK, tmV;
  if (!make_tmap_3d(&tmQ, q, D, H, T, D, ld_q, 64, 128)) return -2;
  if (!make_tmap_3d(&tmK, k_pool, D, G, num_slots, D, (long long)G * D, 64, AW_KV)) return -2;
  if (!make_tmap_3d(&tmV, v_pool, V, G, num_slots, V, (long long)G * V, 64, AW_KV)) return -2;
  AttnWindowParams p = {};
  p.blocks = blocks; p.out = (uint16_t*)out; p.ld_out = ld_out; p.gate = (const uint16_t*)gate; p.ld_gate = ld_gate;
  p.D = D; p.V = V; p.window = window; p.chunk = chunk; p.group = H / G;
  p.page_table = page_table; p.max_pages = max_pages; p.num_pages = (int)(num_slots / 128);
  p.score_bias = score_bias; p.cos_v = cos_v; p.sin_v = sin_v; p.rot_v = rot_v; p.tab_rows = tab_rows;
  p.keep = window > 0 ? keep : 0; p.sinks = sinks; p.head_gate = head_gate; p.ld_head_gate = ld_head_gate;
  if (softcap > 0.f) {
    const double k = (double)scale / softcap;                 // x = k s
    p.cap_log2 = softcap * 1.4426950408889634f;
    p.cap_in = (float)(2.0 * 1.4426950408889634 * k);
    p.cap_lim = k > 1e-3 && k < 1e3 ? (float)(AW_TANH_LIM / k) : -1.f;       // (beyond: the folded coefficients leave fp32's range)
    double f = 1.4426950408889634 * scale;
    for (int i = 0; i < 6; ++i, f *= k * k) p.cap_p[i] = (float)(AW_TANH[i] * f);
  }
  return launch_window(tmQ, tmK, tmV, tmQ, tmK, p, n_blocks, H, scale, dtype, reinterpret_cast<cudaStream_t>(stream_));
}
