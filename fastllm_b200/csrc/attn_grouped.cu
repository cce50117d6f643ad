// Paged grouped-query decode attention for sm_100a with any head widths up to 256 (multiples of 8), a chunk mask or a sliding window
// (which may keep the first tokens of the sequence), soft-capped scores, a sink per head in the softmax or sigmoid weights in its place,
// outputs turned back by the query's position, and an output gate (one per element, or one per head).  Page length 128.
//
// As in attn_decode.cu (head width 128) a page of one key / value head is a full UMMA tile:
//     S^T[128 keys x 16 heads] = K_page[128 x D] * Q^T        64-column tiles, K-major, SW128
//     O^T[V dims   x 16 heads] = V_page^T * P^T               row blocks of 128 dims, A read MN-major
// Rows and heads come through 3-D maps bounded per head, so the tail of a 64-column tile is zero and a head may be narrower than a
// tile.  Work items are the (row, page) pairs a query sees, times key / value heads, times groups of 16 query heads; CTAs stride over
// them (as many per SM as the shared memory of a stage allows, so that one streams pages while another is in its softmax), write
// un-normalised partial outputs with (max, sum), and a combine kernel merges a query's partials, adds the sink's term to the
// denominator and applies o * sigmoid(gate).  Sigmoid weights need no maximum and no denominator: partials are added up.  Kept first tokens are pages of their own in the work list, before the window's.
//
// Every row is its own request (its own page-table row and length), so decoded tokens and short portions of prompts share a launch.
// Page pools must hold finite values everywhere: unused keys of a page are multiplied by P = 0.
#include "ptx.cuh"
#include "launch.h"
#include "tmap.h"

FB_DEFINE_ERROR_API(attn_grouped)

namespace fb {

constexpr int KID_ATTN_GROUPED = 17;
constexpr int AG_PAGE = 128;
constexpr int AG_N = 16;                             // MMA N: query heads per item (padded)
constexpr int AG_TILE = AG_PAGE * 64 * 2;            // 16 KB: [128 keys x 64 columns]
constexpr int AG_QTILE = AG_N * 64 * 2;              // 2 KB
constexpr int AG_P_BYTES = AG_N * AG_PAGE * 2;       // 4 KB
constexpr int AG_TMEM_COLS = 64;                     // S: [0,16)  O blocks: [16 + 16 blk, +16)

struct AttnGroupedParams {
  const int* work;        // [n_work][2] = (row, page index within its request)
  const int* n_work;
  const int* page_table; int max_pages, num_pages;
  const int* kv_lens;
  float* part_o;          // [B, G, splits, H / G, V]
  float* part_ml;         // [B, G, splits, H / G, 2]
  int B, H, G, D, V, dt, vt, splits, max_items, window, chunk, keep;
  float scale_log2;
  float cap_log2, cap_in;     // soft cap c: score = c tanh(scale s / c), in log2 units c log2(e); cap_in = 2 log2(e) scale / c (0: no cap)
  const float* sinks;         // [H] or null
  const float* score_bias;    // [H]: the weight of a key is sigmoid(score + score_bias[h]) (null: softmax)
  const float* cos_v; const float* sin_v;      // [tab_rows, rot_v / 2]: output pairs (2m, 2m + 1) are turned back by the position
  int rot_v, tab_rows;
  uint32_t idesc_s, idesc_o;
};

// first key the query at position n - 1 sees
__device__ __forceinline__ int ag_first(int n, int window, int chunk) {
  if (n <= 0) return 0;
  if (chunk > 0) return (n - 1) - (n - 1) % chunk;
  return window > 0 && n > window ? n - window : 0;
}

// MODE (below): 0 plain softmax; 1 soft cap, kept tokens, sinks, head gates and turned outputs are looked at; 2 sigmoid weights, with all
// of these but sinks.
// pages of the kept first tokens (those before the page where the window starts), and the window's first page
template <int MODE>
__device__ __forceinline__ int ag_kept_pages(int n, int window, int chunk, int keep, int& first_page) {
  first_page = ag_first(n, window, chunk) / AG_PAGE;
  if (MODE == 0) return 0;
  const int kp = (keep + AG_PAGE - 1) / AG_PAGE;
  return kp < first_page ? kp : first_page;
}

// c tanh(x): 1 - 2 / (1 + e^2x) is exact to an fp32 rounding of one, which is all that a score needs
__device__ __forceinline__ float ag_score(const AttnGroupedParams& p, float s) {
  if (p.cap_in == 0.f) return s * p.scale_log2;
  return p.cap_log2 - __fdividef(2.f * p.cap_log2, 1.f + exp2f(s * p.cap_in));
}

// one CTA, B <= 1024: the pages of the kept tokens and those between a row's first and last visible key
__global__ void attn_grouped_plan_kernel(const int* __restrict__ kv_lens, int B, int window, int chunk, int keep, int* __restrict__ work,
                                         int* __restrict__ n_work, int max_items) {
  __shared__ int offs[1025];
  pdl_launch_dependents();
  pdl_wait();
  const int t = threadIdx.x;
  int np = 0, first = 0, kept = 0;
  if (t < B) {
    const int n = kv_lens[t];
    kept = ag_kept_pages<1>(n, window, chunk, keep, first);
    np = n > 0 ? kept + (n + AG_PAGE - 1) / AG_PAGE - first : 0;
  }
  offs[t + 1] = np;
  if (t == 0) offs[0] = 0;
  __syncthreads();
  for (int d = 1; d < blockDim.x; d <<= 1) {
    const int v = t >= d ? offs[t + 1 - d] : 0;
    __syncthreads();
    if (t >= d) offs[t + 1] += v;
    __syncthreads();
  }
  if (t < B) {
    const int base = offs[t];
    for (int i = 0; i < np; ++i)
      if (base + i < max_items) { work[2 * (base + i)] = t; work[2 * (base + i) + 1] = i < kept ? i : first + i - kept; }
  }
  if (t == 0) *n_work = min(offs[blockDim.x], max_items);
}

// Reads and validates one item; every warp role uses this, so a rejected item is rejected by all of them alike.
template <int MODE>
__device__ __forceinline__ bool ag_item(const AttnGroupedParams& p, int w, int& b, int& pg, int& split, int& kvh, int& h0) {
  const int hgs = (p.H / p.G + AG_N - 1) / AG_N, per = p.G * hgs;
  const int item = w / per, r = w - item * per;
  kvh = r / hgs;
  h0 = (r - kvh * hgs) * AG_N;                       // first query head of the item within the key / value head's group
  b = p.work[2 * item]; pg = p.work[2 * item + 1];
  bool ok = (unsigned)b < (unsigned)p.B && (unsigned)pg < (unsigned)p.max_pages;
  if (!ok) { b = 0; pg = 0; }
  int first;
  const int kept = ag_kept_pages<MODE>(p.kv_lens[b], p.window, p.chunk, p.keep, first);
  split = MODE != 0 && pg < kept ? pg : kept + pg - first;
  if ((unsigned)split >= (unsigned)p.splits) { split = 0; ok = false; }
  return ok;
}

template <bool BF16, int GP, int MODE>
__global__ void __launch_bounds__(192, 3)
attn_grouped_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                    const AttnGroupedParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int dt = p.dt, vt = p.vt, vblocks = (vt + 1) >> 1;
  uint8_t* k_smem = smem;
  uint8_t* v_smem = k_smem + dt * AG_TILE;                     // an odd last half block reads one tile past the values: allocated
  uint8_t* q_smem = v_smem + 2 * vblocks * AG_TILE;
  uint8_t* p_smem = q_smem + dt * AG_QTILE;
  uint64_t* bars = reinterpret_cast<uint64_t*>(p_smem + AG_P_BYTES);
  uint64_t* full_k = bars;
  uint64_t* full_v = bars + 1;
  uint64_t* empty_k = bars + 2;
  uint64_t* empty_v = bars + 3;
  uint64_t* s_full = bars + 4;
  uint64_t* p_ready = bars + 5;
  uint64_t* o_full = bars + 6;
  uint64_t* o_empty = bars + 7;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
  float* red_max = reinterpret_cast<float*>(tmem_slot + 4);    // [4 warps][16]
  float* red_sum = red_max + 64;                                // [4 warps][16]

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  bool dead = false;
  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    mbar_init(full_k, 1); mbar_init(full_v, 1); mbar_init(empty_k, 1); mbar_init(empty_v, 1);
    mbar_init(s_full, 1); mbar_init(p_ready, 128); mbar_init(o_full, 1); mbar_init(o_empty, 128);
    mbar_init_fence();
    tma_prefetch_desc(&tmQ); tma_prefetch_desc(&tmK); tma_prefetch_desc(&tmV);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, AG_TMEM_COLS); tmem_relinquish(); }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_s = *tmem_slot;
  const uint32_t tmem_o = tmem_s + 16;
  pdl_wait();
  int n_items = *p.n_work;
  if (n_items < 0) n_items = 0;
  if (n_items > p.max_items) n_items = p.max_items;
  const int HG = p.H / p.G;
  const int total = n_items * p.G * ((HG + AG_N - 1) / AG_N);

  if (warp == 0) {
    if (elect_one()) {
      int it = 0;
      for (int w = blockIdx.x; w < total; w += gridDim.x, ++it) {
        int b, pg, split, kvh, h0;
        if (!ag_item<MODE>(p, w, b, pg, split, kvh, h0)) report_error(ERR_BAD_ARG, KID_ATTN_GROUPED, 20);
        int page = p.page_table[(size_t)b * p.max_pages + pg];
        if ((unsigned)page >= (unsigned)p.num_pages) { report_error(ERR_BAD_ARG, KID_ATTN_GROUPED, 21); page = 0; }
        const uint32_t ph = (uint32_t)it & 1u;
        if (!mbar_wait(empty_k, ph ^ 1u, dead, KID_ATTN_GROUPED, 1)) break;
        mbar_expect_tx(full_k, dt * (AG_TILE + AG_QTILE));
        for (int j = 0; j < dt; ++j) {
          tma_load_3d(k_smem + j * AG_TILE, &tmK, full_k, j * 64, kvh, page * AG_PAGE);
          tma_load_3d(q_smem + j * AG_QTILE, &tmQ, full_k, j * 64, b, kvh * HG + h0);
        }
        if (!mbar_wait(empty_v, ph ^ 1u, dead, KID_ATTN_GROUPED, 2)) break;
        mbar_expect_tx(full_v, vt * AG_TILE);
        for (int j = 0; j < vt; ++j) tma_load_3d(v_smem + j * AG_TILE, &tmV, full_v, j * 64, kvh, page * AG_PAGE);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (elect_one()) {
      const uint32_t kb = smem_u32(k_smem), vb = smem_u32(v_smem), qb = smem_u32(q_smem), pb = smem_u32(p_smem);
      const int ks = (p.D + 15) / 16;
      int it = 0;
      for (int w = blockIdx.x; w < total; w += gridDim.x, ++it) {
        const uint32_t ph = (uint32_t)it & 1u;
        if (!mbar_wait(full_k, ph, dead, KID_ATTN_GROUPED, 3)) break;
        tc_fence_after_sync();
        for (int k = 0; k < ks; ++k)
          umma_f16(tmem_s, make_smem_desc(kb + (k >> 2) * AG_TILE + (k & 3) * 32, 16, 1024, SWZ_128B),
                   make_smem_desc(qb + (k >> 2) * AG_QTILE + (k & 3) * 32, 16, 1024, SWZ_128B), p.idesc_s, k != 0 ? 1u : 0u);
        umma_commit(s_full);
        umma_commit(empty_k);
        if (!mbar_wait(p_ready, ph, dead, KID_ATTN_GROUPED, 4)) break;
        if (!mbar_wait(full_v, ph, dead, KID_ATTN_GROUPED, 5)) break;
        if (it > 0 && !mbar_wait(o_empty, ph ^ 1u, dead, KID_ATTN_GROUPED, 6)) break;
        tc_fence_after_sync();
        for (int blk = 0; blk < vblocks; ++blk) {
#pragma unroll
          for (int k = 0; k < 8; ++k)
            umma_f16(tmem_o + blk * 16, make_smem_desc(vb + 2 * blk * AG_TILE + k * 2048, AG_TILE, 1024, SWZ_128B),
                     make_smem_desc(pb + k * 512, 256, 128, SWZ_NONE), p.idesc_o, k != 0 ? 1u : 0u);
        }
        umma_commit(o_full);
        umma_commit(empty_v);
      }
    }
    __syncwarp();
  } else {
    const int q = warp & 3;                // TMEM lane quarter
    const int t = q * 32 + lane;           // key within the page (softmax) / dim within a block (epilogue)
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    int it = 0;
    for (int w = blockIdx.x; w < total; w += gridDim.x, ++it) {
      int b, pg, split, kvh, h0;
      ag_item<MODE>(p, w, b, pg, split, kvh, h0);
      const int n = p.kv_lens[b], nh = min(GP, HG - h0);
      const uint32_t ph = (uint32_t)it & 1u;
      const int key = pg * AG_PAGE + t;
      const bool valid = key < n && (key >= ag_first(n, p.window, p.chunk) || (MODE != 0 && key < p.keep));
      mbar_wait(s_full, ph, dead, KID_ATTN_GROUPED, 7);
      tc_fence_after_sync();
      uint32_t r[16];
      tmem_ld_32x32b_x16(tmem_s + lane_off, r);
      tmem_ld_wait();
      // P^T[head][key] in the K-major core-matrix layout: ((t/8)*2 + h/8)*128 + (h%8)*16 + (t%8)*2 bytes
      uint8_t* pb = p_smem + (t >> 3) * 256 + (t & 7) * 2;
      if (MODE == 2) {
#pragma unroll
        for (int h = 0; h < 16; ++h) {
          uint16_t bits = 0;
          if (h < GP && h < nh && valid) {
            const float x = ag_score(p, __uint_as_float(r[h])) + p.score_bias[kvh * HG + h0 + h] * 1.4426950408889634f;
            const float pv = __fdividef(1.f, 1.f + exp2f(-x));
            bits = BF16 ? __bfloat16_as_ushort(__float2bfloat16_rn(pv)) : __half_as_ushort(__float2half_rn(pv));
          }
          if (h < GP || it == 0) *reinterpret_cast<uint16_t*>(pb + (h >> 3) * 128 + (h & 7) * 16) = bits;    // unused rows: zeroed once
        }
      } else {
        float sv[GP];
#pragma unroll
        for (int h = 0; h < GP; ++h) {
          sv[h] = (valid && h < nh) ? (MODE != 0 ? ag_score(p, __uint_as_float(r[h])) : __uint_as_float(r[h]) * p.scale_log2) : -INFINITY;
          float m = sv[h];
#pragma unroll
          for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
          if (lane == 0) red_max[q * 16 + h] = m;
        }
        asm volatile("bar.sync 1, 128;\n" ::: "memory");
#pragma unroll
        for (int h = 0; h < 16; ++h) {
          uint16_t bits = 0;
          if (h < GP) {
            const float mx = fmaxf(fmaxf(red_max[h], red_max[16 + h]), fmaxf(red_max[32 + h], red_max[48 + h]));
            const float pv = (h < nh && valid) ? exp2f(sv[h < GP ? h : 0] - mx) : 0.f;
            bits = BF16 ? __bfloat16_as_ushort(__float2bfloat16_rn(pv)) : __half_as_ushort(__float2half_rn(pv));
            // the sum of what the tensor core will see
            float pr = BF16 ? __bfloat162float(__ushort_as_bfloat16(bits)) : __half2float(__ushort_as_half(bits));
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) pr += __shfl_xor_sync(0xffffffffu, pr, o);
            if (lane == 0) red_sum[q * 16 + h] = pr;
          }
          if (h < GP || it == 0) *reinterpret_cast<uint16_t*>(pb + (h >> 3) * 128 + (h & 7) * 16) = bits;      // unused rows: zeroed once
        }
      }
      fence_proxy_async_smem();
      tc_fence_before_sync();
      mbar_arrive(p_ready);
      mbar_wait(o_full, ph, dead, KID_ATTN_GROUPED, 8);
      tc_fence_after_sync();
      const size_t slot = ((size_t)(b * p.G + kvh) * p.splits + split) * HG + h0;
      for (int blk = 0; blk < vblocks; ++blk) {
        tmem_ld_32x32b_x16(tmem_o + blk * 16 + lane_off, r);
        tmem_ld_wait();
        const int d = blk * 128 + t;
        if (d < p.V) {
          float* po = p.part_o + slot * p.V + d;
#pragma unroll
          for (int h = 0; h < GP; ++h)
            if (h < nh) po[(size_t)h * p.V] = __uint_as_float(r[h]);
        }
      }
      tc_fence_before_sync();
      mbar_arrive(o_empty);
      if (MODE != 2 && t < nh) {
        p.part_ml[(slot + t) * 2] = fmaxf(fmaxf(red_max[t], red_max[16 + t]), fmaxf(red_max[32 + t], red_max[48 + t]));
        p.part_ml[(slot + t) * 2 + 1] = red_sum[t] + red_sum[16 + t] + red_sum[32 + t] + red_sum[48 + t];
      }
      if (MODE != 2) asm volatile("bar.sync 1, 128;\n" ::: "memory");     // red_max / red_sum are rewritten by the next item
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_s, AG_TMEM_COLS);
}

// one CTA per (row, query head): merges the row's partials, eight at a time, then sink, rotation and gate
template <bool BF16, int MODE>
__global__ void __launch_bounds__(128) attn_grouped_combine_kernel(const AttnGroupedParams p, uint16_t* __restrict__ out, long long ld_out,
                                                                   const uint16_t* __restrict__ gate, long long ld_gate,
                                                                   const float* __restrict__ head_gate, long long ld_head_gate) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y, HG = p.H / p.G, kvh = h / HG, g = h - kvh * HG;
  const int n = p.kv_lens[b];
  int first;
  const int kept = ag_kept_pages<MODE>(n, p.window, p.chunk, p.keep, first);
  int ns = n > 0 ? kept + (n + AG_PAGE - 1) / AG_PAGE - first : 0;
  if (ns > p.splits) {
    ns = p.splits;
    if (threadIdx.x == 0) report_error(ERR_BAD_ARG, KID_ATTN_GROUPED, 22);
  }
  const size_t base = (size_t)(b * p.G + kvh) * p.splits;
  const float sink = MODE == 1 && p.sinks != nullptr ? p.sinks[h] * 1.4426950408889634f : -INFINITY;
  const float hg = MODE != 0 && head_gate != nullptr ? 1.0f / (1.0f + __expf(-head_gate[(size_t)b * ld_head_gate + h])) : 1.0f;
  const int at = MODE != 0 ? max(0, min(n, p.tab_rows) - 1) : 0;
  for (int d0 = 0; d0 < p.V; d0 += 128) {                // (all lanes stay in the loop: they exchange their halves of a pair)
    const int dd = d0 + threadIdx.x, d = dd < p.V ? dd : p.V - 1;
    float M = -INFINITY, L = 0.f, acc = 0.f;
    for (int s = 0; s < ns; s += 8) {
      float m8[8], l8[8], o8[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        if (s + j < ns) {
          const size_t sl = (base + s + j) * HG + g;
          if (MODE != 2) {
            m8[j] = p.part_ml[sl * 2];
            l8[j] = p.part_ml[sl * 2 + 1];
          }
          o8[j] = p.part_o[sl * p.V + d];
        }
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        if (MODE == 2) {
          if (s + j < ns) acc += o8[j];
        } else if (s + j < ns) {
          const float nm = fmaxf(M, m8[j]);
          if (nm > -INFINITY) {
            const float a = exp2f(M - nm), bw = exp2f(m8[j] - nm);
            acc = acc * a + o8[j] * bw;
            L = L * a + l8[j] * bw;
            M = nm;
          }
        }
      }
    }
    if (MODE == 1 && sink > -INFINITY && L > 0.f) {
      const float nm = fmaxf(M, sink), a = exp2f(M - nm);
      acc *= a;
      L = L * a + exp2f(sink - nm);
    }
    float o = MODE == 2 ? acc * hg : L > 0.f ? (MODE == 1 ? acc / L * hg : acc / L) : 0.f;
    if (MODE != 0 && p.rot_v > 0) {
      const float other = __shfl_xor_sync(0xffffffffu, o, 1);
      if (dd < p.rot_v) {
        const size_t e = (size_t)at * (p.rot_v >> 1) + (dd >> 1);
        o = o * p.cos_v[e] + ((dd & 1) ? -other : other) * p.sin_v[e];
      }
    }
    if (dd >= p.V) continue;
    if (gate != nullptr) {
      const uint16_t gb = gate[(size_t)b * ld_gate + (size_t)h * p.V + d];
      const float gv = BF16 ? __bfloat162float(__ushort_as_bfloat16(gb)) : __half2float(__ushort_as_half(gb));
      o *= 1.0f / (1.0f + __expf(-gv));
    }
    out[(size_t)b * ld_out + (size_t)h * p.V + d] = BF16 ? __bfloat16_as_ushort(__float2bfloat16_rn(o)) : __half_as_ushort(__float2half_rn(o));
  }
}

}  // namespace fb

using namespace fb;

// work: [2 * max_items] ints, n_work: [1].
extern "C" int fb_grouped_plan(const int* kv_lens, int B, int window, int chunk, int keep, int* work, int* n_work, int max_items, void* stream) {
  if (B <= 0 || B > 1024 || max_items <= 0 || window < 0 || chunk < 0 || keep < 0) return -1;
  int threads = 32;
  while (threads < B) threads <<= 1;
  launch_k(attn_grouped_plan_kernel, dim3(1), dim3(threads), 0, reinterpret_cast<cudaStream_t>(stream), 0, kv_lens, B, window, chunk, keep, work, n_work, max_items);
  return (int)cudaGetLastError();
}

// score_bias [H] (null: softmax): see AttnGroupedParams; rot_v > 0: outputs are turned back by the row's position, tables [tab_rows, rot_v / 2].
// keep: first tokens a window keeps; softcap 0: none; sinks [H], head_gate (row stride ld_head_gate, one logit per head): null for none.
// q: [B, >= H * D] (row stride ld_q), k_pool [num_slots, G, D], v_pool [num_slots, G, V], out / gate [B, >= H * V]; 16-bit (dtype 0 = fp16,
// 1 = bf16).  splits: most pages one query's keys touch; part_o [B * H * splits * V], part_ml [B * H * splits * 2] floats.
extern "C" int fb_grouped_decode(const void* q, long long ld_q, const void* k_pool, const void* v_pool, void* out, long long ld_out,
                                 const void* gate, long long ld_gate, const int* page_table, const int* kv_lens, const int* work,
                                 const int* n_work, float* part_o, float* part_ml, int B, int H, int G, int D, int V, long long num_slots,
                                 int max_pages, int splits, int max_items, int window, int chunk, int keep, float scale, float softcap,
                                 const float* sinks, const float* head_gate, long long ld_head_gate, const float* score_bias, const float* cos_v,
                                 const float* sin_v, int rot_v, int tab_rows, int dtype, void* stream_) {
  if (B <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G != 0 || H > 65535 || D <= 0 || V <= 0 || D > 256 || V > 256 || D % 8 != 0 || V % 8 != 0 || num_slots < AG_PAGE ||
      max_pages <= 0 || splits <= 0 || keep < 0 || softcap < 0.f || (dtype != 0 && dtype != 1) || rot_v < 0 || (rot_v & 1) || rot_v > V || (score_bias != nullptr && sinks != nullptr) ||
      (rot_v > 0 && (cos_v == nullptr || sin_v == nullptr || tab_rows <= 0)))
    return -1;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  static int sm_count = 0;
  if (sm_count == 0) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sm_count, cudaDevAttrMultiProcessorCount, dev);
  }
  CUtensorMap tmQ, tmK, tmV;
  if (!make_tmap_3d(&tmQ, q, D, B, H, ld_q, D, 64, AG_N)) return -2;
  if (!make_tmap_3d(&tmK, k_pool, D, G, num_slots, D, (long long)G * D, 64, AG_PAGE)) return -2;
  if (!make_tmap_3d(&tmV, v_pool, V, G, num_slots, V, (long long)G * V, 64, AG_PAGE)) return -2;
  AttnGroupedParams p;
  p.work = work; p.n_work = n_work; p.page_table = page_table; p.max_pages = max_pages; p.num_pages = (int)(num_slots / AG_PAGE);
  p.kv_lens = kv_lens; p.part_o = part_o; p.part_ml = part_ml;
  p.B = B; p.H = H; p.G = G; p.D = D; p.V = V; p.dt = (D + 63) / 64; p.vt = (V + 63) / 64; p.splits = splits; p.max_items = max_items;
  p.window = window; p.chunk = chunk; p.keep = keep; p.scale_log2 = scale * 1.4426950408889634f;
  p.cap_log2 = softcap * 1.4426950408889634f; p.cap_in = softcap > 0.f ? 2.f * 1.4426950408889634f * scale / softcap : 0.f;
  p.sinks = sinks; p.score_bias = score_bias; p.cos_v = cos_v; p.sin_v = sin_v; p.rot_v = rot_v; p.tab_rows = tab_rows;
  const uint32_t f = dtype == 1 ? 1u : 0u;
  p.idesc_s = make_idesc(f, f, 0, 0, 128, AG_N);
  p.idesc_o = make_idesc(f, f, 1, 0, 128, AG_N);
  const int smem = (p.dt + 2 * ((p.vt + 1) / 2)) * AG_TILE + p.dt * AG_QTILE + AG_P_BYTES + 1024 + 1024;
  int occ = (227 * 1024) / (smem + 1024);
  occ = occ < 1 ? 1 : occ > 3 ? 3 : occ;
  const int HG = H / G, gp = HG >= 16 ? 16 : HG;
  const int mode = score_bias != nullptr ? 2 : keep > 0 || softcap > 0.f || sinks != nullptr || head_gate != nullptr || rot_v > 0 ? 1 : 0;
#define FB_AG(BF, GPV, MODE)                                                                                                         \
  {                                                                                                                                  \
    static DeviceOnce cfg;                                                                                                           \
    if (cfg.need()) cudaFuncSetAttribute(attn_grouped_kernel<BF, GPV, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024); \
    launch_k<PDL_ATTN>(attn_grouped_kernel<BF, GPV, MODE>, dim3(sm_count * occ), dim3(192), smem, stream, 0, tmQ, tmK, tmV, p);        \
  }
#define FB_AG_GP(BF, MODE)                                                                                                           \
  {                                                                                                                                  \
    if (gp <= 1) FB_AG(BF, 1, MODE) else if (gp <= 2) FB_AG(BF, 2, MODE) else if (gp <= 4) FB_AG(BF, 4, MODE)                            \
    else if (gp <= 8) FB_AG(BF, 8, MODE) else FB_AG(BF, 16, MODE)                                                                      \
    launch_k<PDL_COMBINE>(attn_grouped_combine_kernel<BF, MODE>, dim3(B, H), dim3(128), 0, stream, 0, p, (uint16_t*)out, ld_out,       \
                          (const uint16_t*)gate, ld_gate, head_gate, ld_head_gate);                                                  \
  }
  if (dtype == 1) { if (mode == 2) FB_AG_GP(true, 2) else if (mode == 1) FB_AG_GP(true, 1) else FB_AG_GP(true, 0) }
  else { if (mode == 2) FB_AG_GP(false, 2) else if (mode == 1) FB_AG_GP(false, 1) else FB_AG_GP(false, 0) }
#undef FB_AG_GP
#undef FB_AG
  return (int)cudaGetLastError();
}
