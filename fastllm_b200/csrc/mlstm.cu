// Matrix-memory LSTM (mLSTM of xLSTM) for sm_100a: per head a [D, V] fp32 state S and a normaliser row n [D] under a running maximum m.
// A token with query q, key k, value v, log input gate i and log forget gate f does
//     m' = max(f + m, i),   S <- e^(f + m - m') S + e^(i - m') k v^T,   n <- e^(f + m - m') n + e^(i - m') k,
//     out = S^T q / (max(|n . q|, e^(-m')) + 1e-6),
// then every head's output is divided by its root mean square, multiplied by a norm weight and by sigmoid(gate).  The gates come from
// fp32 logits: i = cap tanh(z_i / cap), f = log sigmoid(cap tanh(z_f / cap)).
//
//  * mlstm_recurrent_kernel: one CTA per (head, request) walks the request's tokens with the state in registers; a thread owns R rows of
//    one state column, so the state is read once and written once per step.  Any widths, fp32 included.
//  * the chunked form for prompts, 128 tokens a chunk.  With F_t the running sum of f inside the chunk, a_s = i_s - F_s and
//    M_t = max(m_0, max_(s <= t) a_s), the recurrence is  m_t = F_t + M_t  and
//        S_t = e^(m_0 - M_t) S_0 + sum_(s <= t) e^(a_s - M_t) k_s v_s^T        (n alike),
//    whose exponents are never positive.  All chunks and heads run in parallel except for the scan:
//      mlstm_chunk_state   U_c = sum_s e^(a_s - A_c) k_s v_s^T,  A_c = max_s a_s    (tcgen05: U^T[V x D] = (w V)^T K over the tokens)
//      mlstm_chunk_scan    carries (S, n, m) over the chunks of a request, leaves every chunk's first state
//      mlstm_chunk_out     O = e^(m_0 - M_t) Q S_0 + (Q K^T * e^(a_s - M_t)) V      (tcgen05, both products into one accumulator)
//    Tensor-core operands are 16 bits wide: queries, keys and values are that already; what has fp32 precision (weighted values,
//    weighted scores, states) enters as two 16-bit terms, the rounded value and the rounded remainder, so products keep 16 bits and
//    more of mantissa.  The state itself is carried in fp32.
//
// Compiled without fast-math.
#include "ptx.cuh"
#include "launch.h"
#include "tmap.h"

FB_DEFINE_ERROR_API(mlstm)

namespace fb {

constexpr int KID_MLSTM = 18;
constexpr float ML_LOG2E = 1.4426950408889634f;
constexpr float ML_LN2 = 0.69314718055994531f;

template <int DT> struct MAct;
template <> struct MAct<0> { typedef uint16_t T; static __device__ __forceinline__ float ld(uint16_t v) { return __half2float(__ushort_as_half(v)); }
                             static __device__ __forceinline__ uint16_t st(float v) { return __half_as_ushort(__float2half_rn(v)); } };
template <> struct MAct<1> { typedef uint16_t T; static __device__ __forceinline__ float ld(uint16_t v) { return __bfloat162float(__ushort_as_bfloat16(v)); }
                             static __device__ __forceinline__ uint16_t st(float v) { return __bfloat16_as_ushort(__float2bfloat16_rn(v)); } };
template <> struct MAct<2> { typedef float T; static __device__ __forceinline__ float ld(float v) { return v; } static __device__ __forceinline__ float st(float v) { return v; } };

struct MlstmParams {
  const void* proj; long long ld;          // [T, ld] rows: queries from column 0, then keys, values, output gate at *_col
  const float* gates; long long ld_gates;  // [T, ld_gates] logits: input gates of the heads, then forget gates
  const float* gate_b;                     // [2 H] their biases
  const void* norm_w;                      // [H * V]
  float* state; long long st_head;         // [slots, H, st_head]: S [D, V], n [D], m
  void* out; long long ld_out;             // [T, >= H * V]
  int H, D, V, k_col, v_col, g_col;
  float scale, cap, eps;
  // recurrent form: one token per request (items null), or (first row, rows, slot) of every request
  const int* slots; const int* items;
  // chunked form over the heads [h0, h0 + Hn); unit = chunk * Hn + head - h0
  const int* chunks;                       // [n_chunks][3] = (first row, rows, state slot if it is the request's last chunk, else -1)
  const int* reqs;                         // [n_reqs][3] = (first chunk, chunks, slot)
  float* inc; float* ninc;                 // [units, D, V], [units, D]
  float* lg;                               // [units][3][128] log2 units: a_s, running maximum of a, F_t
  float* m0; float* n0;                    // [units] (log2 units), [units, D]
  uint16_t* s0;                            // [units][2][Dp, V]: the two terms of S_0
  int n_chunks, h0, Hn, Dp;
};

__device__ __forceinline__ float ml_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float ml_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ void ml_gates(const MlstmParams& p, int t, int h, float& i, float& f) {
  const float* z = p.gates + (size_t)t * p.ld_gates + h;
  i = p.cap * tanhf((z[0] + p.gate_b[h]) / p.cap);
  f = ml_log_sigmoid(p.cap * tanhf((z[p.H] + p.gate_b[p.H + h]) / p.cap));
}

// ------------------------------------------------------------------------------------------------
// recurrent form
// ------------------------------------------------------------------------------------------------
// Threads: ceil(V / 32) column groups x row groups of R rows; R = 0: the state stays in memory (widths beyond the register forms).
template <int DT, int R>
__global__ void __launch_bounds__(512) mlstm_recurrent_kernel(const MlstmParams p, int row_groups) {
  typedef typename MAct<DT>::T T;
  extern __shared__ float sm[];
  const int D = p.D, V = p.V, tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31, nw = nt >> 5;
  const int cgs = (V + 31) >> 5;
  const int rows = R > 0 ? R : (D + row_groups - 1) / row_groups, Dp = (rows * row_groups + 3) & ~3;
  float* qs = sm;                    // [Dp] (zero beyond D)
  float* ks = qs + Dp;               // [Dp] keys times the input gate
  float* ns = ks + Dp;               // [Dp]
  float* part = ns + Dp;             // [row_groups][32 * cgs]
  float* red = part + row_groups * 32 * cgs;     // [2][16]
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y;
  const int t0 = p.items != nullptr ? p.items[3 * b] : b, cnt = p.items != nullptr ? p.items[3 * b + 1] : 1;
  const int slot = p.items != nullptr ? p.items[3 * b + 2] : p.slots[b];
  if (cnt <= 0) return;
  const int cg = warp % cgs, rg = warp / cgs, j = cg * 32 + lane;
  const bool col = j < V;
  float* S = p.state + ((size_t)slot * p.H + h) * p.st_head;
  float* N = S + (size_t)D * V;
  float m = N[D];
  const int r0 = rg * rows, rn = min(rows, D - r0);
  // every load of a token is requested before the first one is waited for: the state, the normaliser (a thread's first element stays in
  // a register), the rows
  float s[R > 0 ? R : 1];
  if (R > 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) s[i] = (col && i < rn) ? S[(size_t)(r0 + i) * V + j] : 0.f;
  }
  float nv = tid < D ? N[tid] : 0.f;
  const T* w = reinterpret_cast<const T*>(p.norm_w) + (size_t)h * V;
  const T wv = w[tid < V ? tid : 0];
  for (int d = tid + nt; d < D; d += nt) ns[d] = N[d];
  for (int d = D + tid; d < Dp; d += nt) { qs[d] = 0.f; ks[d] = 0.f; }
  for (int t = t0; t < t0 + cnt; ++t) {
    const T* row = reinterpret_cast<const T*>(p.proj) + (size_t)t * p.ld;
    const int d0 = h * D + (tid < D ? tid : 0), v0 = h * V + (tid < V ? tid : 0);
    const T qr = row[d0], kr = row[p.k_col + d0], gr = row[p.g_col + v0], vr = row[p.v_col + h * V + (col ? j : 0)];
    float ig, fg;
    ml_gates(p, t, h, ig, fg);
    const float mn = fmaxf(fg + m, ig), keep = expf(fg + m - mn), add = expf(ig - mn);
    m = mn;
    float dot = 0.f;
    for (int d = tid; d < D; d += nt) {
      const bool own = d == tid;
      const float q = MAct<DT>::ld(own ? qr : row[h * D + d]) * p.scale, k = MAct<DT>::ld(own ? kr : row[p.k_col + h * D + d]) * add;
      const float n = fmaf(own ? nv : ns[d], keep, k);
      qs[d] = q; ks[d] = k;
      if (own) nv = n; else ns[d] = n;
      dot = fmaf(n, q, dot);
    }
    const float v = col ? MAct<DT>::ld(vr) : 0.f;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
    if (lane == 0) red[warp] = dot;
    __syncthreads();
    float o = 0.f;
    if (R > 0) {
      const float4 *k4 = reinterpret_cast<const float4*>(ks + r0), *q4 = reinterpret_cast<const float4*>(qs + r0);
#pragma unroll
      for (int i = 0; i < R / 4; ++i) {
        const float4 kk = k4[i], qq = q4[i];
        s[4 * i] = fmaf(s[4 * i], keep, kk.x * v); s[4 * i + 1] = fmaf(s[4 * i + 1], keep, kk.y * v);
        s[4 * i + 2] = fmaf(s[4 * i + 2], keep, kk.z * v); s[4 * i + 3] = fmaf(s[4 * i + 3], keep, kk.w * v);
        o = fmaf(s[4 * i], qq.x, o); o = fmaf(s[4 * i + 1], qq.y, o); o = fmaf(s[4 * i + 2], qq.z, o); o = fmaf(s[4 * i + 3], qq.w, o);
        if ((i & 3) == 3) asm volatile("" ::: "memory");       // keeps the reads of a few rows in flight, not of all of them
      }
    } else if (col) {
      for (int i = 0; i < rn; ++i) {
        float* sp = S + (size_t)(r0 + i) * V + j;
        const float x = fmaf(*sp, keep, ks[r0 + i] * v);
        *sp = x;
        o = fmaf(x, qs[r0 + i], o);
      }
    }
    part[rg * 32 * cgs + j] = o;
    dot = 0.f;
    for (int x = 0; x < nw; ++x) dot += red[x];
    const float den = fmaxf(fabsf(dot), expf(-m)) + 1e-6f;
    __syncthreads();
    // output of the head: sum over the row groups, its root mean square, norm weight, gate
    float ss = 0.f;
    for (int i = tid; i < V; i += nt) {
      float x = part[i];
      for (int g = 1; g < row_groups; ++g) x += part[g * 32 * cgs + i];
      x /= den;
      part[i] = x;
      ss += x * x;
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    if (lane == 0) red[16 + warp] = ss;
    __syncthreads();
    ss = 0.f;
    for (int x = 0; x < nw; ++x) ss += red[16 + x];
    const float inv = 1.0f / sqrtf(ss / (float)V + p.eps);
    for (int i = tid; i < V; i += nt) {
      const float g = MAct<DT>::ld(i == tid ? gr : row[p.g_col + h * V + i]), wi = MAct<DT>::ld(i == tid ? wv : w[i]);
      reinterpret_cast<T*>(p.out)[(size_t)t * p.ld_out + (size_t)h * V + i] = MAct<DT>::st(part[i] * inv * wi / (1.0f + expf(-g)));
    }
    __syncthreads();                     // part / red / qs are rewritten by the next token
  }
  for (int d = tid; d < D; d += nt) N[d] = d == tid ? nv : ns[d];
  if (tid == 0) N[D] = m;
  if (R > 0 && col) {
    int step = V;
    asm volatile("" : "+r"(step));       // new addresses: those of the loads need not stay alive over the token loop
    float* sp = S + (size_t)r0 * step + j;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      if (i < rn) *sp = s[i];
      sp += step;
    }
  }
}

// ------------------------------------------------------------------------------------------------
// chunked form
// ------------------------------------------------------------------------------------------------
constexpr int MC = 128;                        // tokens per chunk
constexpr int MC_TILE = MC * 128;              // 16 KB: [128 rows x 64 columns], 128-byte swizzle
constexpr int MC_STATE_THREADS = 256;
constexpr int MC_SMEM_MAX = 227 * 1024;

// byte offset of 16-byte unit `u` (8 columns) of row `r` in a swizzled [rows x 64] tile
__device__ __forceinline__ int ml_swz(int r, int u) { return r * 128 + ((u ^ (r & 7)) << 4); }

template <bool BF16>
__device__ __forceinline__ void ml_split8(const float* x, uint4& hi, uint4& lo) {
  uint32_t a[4], b[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    a[i] = pack_16<BF16>(x[2 * i], x[2 * i + 1]);
    const float2 f = unpack_16<BF16>(a[i]);
    b[i] = pack_16<BF16>(x[2 * i] - f.x, x[2 * i + 1] - f.y);
  }
  hi = make_uint4(a[0], a[1], a[2], a[3]);
  lo = make_uint4(b[0], b[1], b[2], b[3]);
}

template <bool BF16>
__global__ void __launch_bounds__(MC_STATE_THREADS, 2) mlstm_chunk_state_kernel(const __grid_constant__ CUtensorMap tmK, const MlstmParams p, int tmem_cols) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int D = p.D, V = p.V, dt = (D + 63) >> 6, vblocks = (V + 127) >> 7, Dn = (D + 15) & ~15;
  uint8_t* k_smem = smem;                                      // [dt] tiles
  uint8_t* hi_smem = k_smem + dt * MC_TILE;                    // [2 vblocks] tiles of weighted values, then their remainders
  uint8_t* lo_smem = hi_smem + 2 * vblocks * MC_TILE;
  float* ws = reinterpret_cast<float*>(lo_smem + 2 * vblocks * MC_TILE);      // [128]
  float* part = ws + MC;                                       // [512]
  float* red = part + 512;                                     // [8]
  uint64_t* full_k = reinterpret_cast<uint64_t*>(red + 8);
  uint64_t* done = full_k + 1;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c = blockIdx.x, hl = blockIdx.y, h = p.h0 + hl;
  const int r0 = p.chunks[3 * c], n = p.chunks[3 * c + 1];
  const size_t unit = (size_t)c * p.Hn + hl;
  bool dead = false;
  if (tid == 0) {
    mbar_init(full_k, 1);
    mbar_init(done, 1);
    mbar_init_fence();
    mbar_expect_tx(full_k, dt * MC_TILE);
    for (int j = 0; j < dt; ++j) tma_load_3d(k_smem + j * MC_TILE, &tmK, full_k, j * 64, h, r0);
  }
  if (warp == 1) { tmem_alloc(tmem_slot, tmem_cols); tmem_relinquish(); }
  // this thread's first values, requested before anything is waited for
  constexpr int PRE = 8;
  const uint16_t* vp = reinterpret_cast<const uint16_t*>(p.proj) + (size_t)r0 * p.ld + p.v_col + (size_t)h * V;
  const int vecs = V >> 3;
  uint4 pre[PRE];
#pragma unroll
  for (int i = 0; i < PRE; ++i) {
    const int at = tid + i * MC_STATE_THREADS, s = at / vecs, u = at - s * vecs;
    pre[i] = s < n ? *reinterpret_cast<const uint4*>(vp + (size_t)s * p.ld + u * 8) : make_uint4(0u, 0u, 0u, 0u);
  }
  // one token a thread: running sum of the log forget gates, then a and its running maximum
  float F = 0.f, a = -INFINITY, pm = -INFINITY;
  if (warp < MC / 32) {
    float ig = -INFINITY;
    if (tid < n) ml_gates(p, r0 + tid, h, ig, F);
    F *= ML_LOG2E;
    a = ig * ML_LOG2E;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, F, o); if (lane >= o) F += x; }
    if (lane == 31) red[warp] = F;
  }
  __syncthreads();
  if (warp < MC / 32) {
    for (int w = 0; w < warp; ++w) F += red[w];
    a -= F;
    pm = a;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, pm, o); if (lane >= o) pm = fmaxf(pm, x); }
    if (lane == 31) red[4 + warp] = pm;
  }
  __syncthreads();
  if (warp < MC / 32) {
    for (int w = 0; w < warp; ++w) pm = fmaxf(pm, red[4 + w]);
    float* lg = p.lg + unit * 3 * MC + tid;
    lg[0] = a; lg[MC] = pm; lg[2 * MC] = F;
    ws[tid] = ml_ex2(a - fmaxf(fmaxf(red[4], red[5]), fmaxf(red[6], red[7])));
  }
  __syncthreads();
  // weighted values, two terms each
  auto put = [&](int s, int u, const uint4& raw) {
    const uint32_t r[4] = {raw.x, raw.y, raw.z, raw.w};
    const float w = ws[s];
    float x[8];
#pragma unroll
    for (int j = 0; j < 4; ++j) { const float2 f = unpack_16<BF16>(r[j]); x[2 * j] = f.x * w; x[2 * j + 1] = f.y * w; }
    uint4 hi, lo;
    ml_split8<BF16>(x, hi, lo);
    const int at = (u >> 3) * MC_TILE + ml_swz(s, u & 7);
    *reinterpret_cast<uint4*>(hi_smem + at) = hi;
    *reinterpret_cast<uint4*>(lo_smem + at) = lo;
  };
#pragma unroll
  for (int i = 0; i < PRE; ++i) {
    const int at = tid + i * MC_STATE_THREADS, s = at / vecs;
    if (s < MC) put(s, at - s * vecs, pre[i]);
  }
  for (int at = tid + PRE * MC_STATE_THREADS; at < MC * vecs; at += MC_STATE_THREADS) {
    const int s = at / vecs, u = at - s * vecs;
    put(s, u, s < n ? *reinterpret_cast<const uint4*>(vp + (size_t)s * p.ld + u * 8) : make_uint4(0u, 0u, 0u, 0u));
  }
  fence_proxy_async_smem();
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *tmem_slot;
  if (warp == 0 && elect_one()) {
    if (mbar_wait(full_k, 0, dead, KID_MLSTM, 1)) {
      const uint32_t kb = smem_u32(k_smem), idesc = make_idesc(BF16 ? 1 : 0, BF16 ? 1 : 0, 1, 1, 128, Dn);
      for (int blk = 0; blk < vblocks; ++blk)
        for (int term = 0; term < 2; ++term) {
          const uint32_t vb = smem_u32(term == 0 ? hi_smem : lo_smem) + 2 * blk * MC_TILE;
          for (int k = 0; k < MC / 16; ++k)
            umma_f16(tmem + blk * Dn, make_smem_desc(vb + k * 2048, MC_TILE, 1024, SWZ_128B), make_smem_desc(kb + k * 2048, MC_TILE, 1024, SWZ_128B), idesc,
                     (term | k) != 0 ? 1u : 0u);
        }
      umma_commit(done);
    }
  }
  __syncwarp();
  // the normaliser's increment on the CUDA cores meanwhile, half of the tokens a thread
  mbar_wait(full_k, 0, dead, KID_MLSTM, 2);
  for (int e = tid; e < 2 * D; e += MC_STATE_THREADS) {
    const int half = e >= D ? 1 : 0, d = e - half * D, u = (d & 63) >> 3, s0 = half * (MC / 2);
    const uint8_t* base = k_smem + (d >> 6) * MC_TILE + (d & 7) * 2;
    float x = 0.f;
#pragma unroll 16
    for (int s = s0; s < s0 + MC / 2; ++s) x = fmaf(MAct<BF16 ? 1 : 0>::ld(*reinterpret_cast<const uint16_t*>(base + ml_swz(s, u))), ws[s], x);
    part[e] = x;                                               // (tokens behind the last one: weight 0, rows of later tokens or zeros)
  }
  __syncthreads();
  for (int d = tid; d < D; d += MC_STATE_THREADS) p.ninc[unit * D + d] = part[d] + part[D + d];
  mbar_wait(done, 0, dead, KID_MLSTM, 3);
  tc_fence_after_sync();
  float* U = p.inc + unit * D * V;
  const int q = warp & 3;
  for (int blk = 0; blk < vblocks; ++blk) {
    const int v = blk * 128 + q * 32 + lane;
    for (int c0 = (warp >> 2) * 16; c0 < Dn; c0 += 32) {
      uint32_t r[16];
      __syncwarp();
      tmem_ld_32x32b_x16(tmem + blk * Dn + c0 + ((uint32_t)(q * 32) << 16), r);
      tmem_ld_wait();
      if (v < V) {
#pragma unroll
        for (int j = 0; j < 16; ++j)
          if (c0 + j < D) U[(size_t)(c0 + j) * V + v] = __uint_as_float(r[j]);
      }
    }
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, tmem_cols);
}

// Two state elements (or normaliser elements, behind them) of a (request, head) per thread; reads run ahead of the dependent chain.
template <bool BF16>
__global__ void __launch_bounds__(128) mlstm_chunk_scan_kernel(const MlstmParams p) {
  const int D = p.D, V = p.V, hl = blockIdx.y;
  const int e = (blockIdx.x * 128 + threadIdx.x) * 2;
  if (e >= D * V + D) return;
  const int c0 = p.reqs[3 * blockIdx.z], n = p.reqs[3 * blockIdx.z + 1], slot = p.reqs[3 * blockIdx.z + 2];
  float* head = p.state + ((size_t)slot * p.H + p.h0 + hl) * p.st_head;
  float2 s = *reinterpret_cast<float2*>(head + e);
  float m = head[D * V + D] * ML_LOG2E;                  // (the stored maximum is rewritten by the kernel after this one)
  const bool norm = e >= D * V;
  const float* U = norm ? p.ninc + (size_t)hl * D + (e - D * V) : p.inc + (size_t)hl * D * V + e;
  const size_t su = (size_t)p.Hn * (norm ? D : D * V);
  U += (size_t)c0 * su;
  const float* lg = p.lg + ((size_t)c0 * p.Hn + hl) * 3 * MC;
  const size_t sl = (size_t)p.Hn * 3 * MC;
  constexpr int A = 8;
  float2 u[2][A];
  float top[2][A], F[2][A];
  auto fetch = [&](int k, int c) {
#pragma unroll
    for (int i = 0; i < A; ++i)
      if (c + i < n) {
        u[k][i] = *reinterpret_cast<const float2*>(U + (size_t)(c + i) * su);
        top[k][i] = lg[(size_t)(c + i) * sl + 2 * MC - 1];
        F[k][i] = lg[(size_t)(c + i) * sl + 3 * MC - 1];
      }
  };
  auto step = [&](int k, int c) {
#pragma unroll
    for (int i = 0; i < A; ++i) {
      if (c + i >= n) break;
      const size_t unit = (size_t)(c0 + c + i) * p.Hn + hl;
      if (norm) {
        *reinterpret_cast<float2*>(p.n0 + unit * D + (e - D * V)) = s;
      } else {
        const uint32_t hi = pack_16<BF16>(s.x, s.y);
        const float2 f = unpack_16<BF16>(hi);
        uint16_t* dst = p.s0 + unit * 2 * p.Dp * V + e;
        *reinterpret_cast<uint32_t*>(dst) = hi;
        *reinterpret_cast<uint32_t*>(dst + (size_t)p.Dp * V) = pack_16<BF16>(s.x - f.x, s.y - f.y);
        if (e == 0) p.m0[unit] = m;
      }
      const float M = fmaxf(m, top[k][i]), keep = ml_ex2(m - M), add = ml_ex2(top[k][i] - M);
      s.x = fmaf(s.x, keep, u[k][i].x * add);
      s.y = fmaf(s.y, keep, u[k][i].y * add);
      m = F[k][i] + M;
    }
  };
  fetch(0, 0);
  for (int c = 0; c < n; c += 2 * A) {
    fetch(1, c + A);
    step(0, c);
    fetch(0, c + 2 * A);
    step(1, c + A);
  }
  *reinterpret_cast<float2*>(head + e) = s;
}

// One chunk of one head: warp 0 loads, warp 1 issues the products, warps 2..9 own the tokens, two threads a token (its columns in
// alternating blocks of 32).  The state's two terms and the values pass through one buffer in turn, the weighted scores take the place of
// queries and keys, so that two CTAs share an SM.
constexpr int MC_OUT_THREADS = 320;
template <bool BF16>
__global__ void __launch_bounds__(MC_OUT_THREADS, 2) mlstm_chunk_out_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                                                                            const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmS,
                                                                            const MlstmParams p, int tmem_cols) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int D = p.D, V = p.V, dt = (D + 63) >> 6, vt = (V + 63) >> 6, Dp = p.Dp, Vn = (V + 15) & ~15;
  const int st = Dp * 128;                                     // bytes of a [Dp x 64] state tile
  uint8_t* q_smem = smem;                                      // [dt] tiles, then keys; later the weighted scores: [2] tiles, their remainders
  uint8_t* k_smem = q_smem + dt * MC_TILE;
  uint8_t* p_smem = smem;
  uint8_t* b_smem = smem + (2 * dt > 4 ? 2 * dt : 4) * MC_TILE;       // [vt] tiles: state, its remainders, values
  float* as = reinterpret_cast<float*>(b_smem + vt * (st > MC_TILE ? st : MC_TILE));      // [128]
  float* n0 = as + MC;                                         // [D <= 256]
  float* red = n0 + 256;                                       // [2][2][128]
  uint64_t* full_qk = reinterpret_cast<uint64_t*>(red + 4 * MC);
  uint64_t* full_b = full_qk + 1;
  uint64_t* b_free = full_qk + 2;
  uint64_t* o_init = full_qk + 3;
  uint64_t* p_ready = full_qk + 4;
  uint64_t* o_full = full_qk + 5;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(full_qk + 6);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int c = blockIdx.x, hl = blockIdx.y, h = p.h0 + hl;
  const int r0 = p.chunks[3 * c], n = p.chunks[3 * c + 1], last_slot = p.chunks[3 * c + 2];
  const size_t unit = (size_t)c * p.Hn + hl;
  bool dead = false;
  if (tid == 0) {
    mbar_init(full_qk, 1); mbar_init(full_b, 1); mbar_init(b_free, 1); mbar_init(o_init, 1); mbar_init(p_ready, 256); mbar_init(o_full, 1);
    mbar_init_fence();
    mbar_expect_tx(full_qk, 2 * dt * MC_TILE);
    for (int j = 0; j < dt; ++j) {
      tma_load_3d(q_smem + j * MC_TILE, &tmQ, full_qk, j * 64, h, r0);
      tma_load_3d(k_smem + j * MC_TILE, &tmK, full_qk, j * 64, h, r0);
    }
    mbar_expect_tx(full_b, vt * st);
    for (int j = 0; j < vt; ++j) tma_load_2d(b_smem + j * st, &tmS, full_b, j * 64, (int)(unit * 2 * Dp));
  }
  if (warp == 1) { tmem_alloc(tmem_slot, tmem_cols); tmem_relinquish(); }
  for (int i = tid; i < D; i += MC_OUT_THREADS) n0[i] = p.n0[unit * D + i];
  for (int i = tid; i < MC; i += MC_OUT_THREADS) as[i] = p.lg[unit * 3 * MC + i];
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + MC;
  if (warp == 0) {
    if (elect_one()) {
      if (mbar_wait(b_free, 0, dead, KID_MLSTM, 11)) {
        mbar_expect_tx(full_b, vt * st);
        for (int j = 0; j < vt; ++j) tma_load_2d(b_smem + j * st, &tmS, full_b, j * 64, (int)((unit * 2 + 1) * Dp));
        if (mbar_wait(b_free, 1, dead, KID_MLSTM, 12)) {
          mbar_expect_tx(full_b, vt * MC_TILE);
          for (int j = 0; j < vt; ++j) tma_load_3d(b_smem + j * MC_TILE, &tmV, full_b, j * 64, h, r0);
        }
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    if (elect_one()) {
      const uint32_t f = BF16 ? 1u : 0u, qb = smem_u32(q_smem), kb = smem_u32(k_smem), bb = smem_u32(b_smem), pb = smem_u32(p_smem);
      const uint32_t id_s = make_idesc(f, f, 0, 0, 128, MC), id_o = make_idesc(f, f, 0, 1, 128, Vn);
      const int ks = Dp >> 4;
      bool ok = mbar_wait(full_qk, 0, dead, KID_MLSTM, 4);
      if (ok) {
        tc_fence_after_sync();
        for (int k = 0; k < ks; ++k)
          umma_f16(tmem_s, make_smem_desc(qb + (k >> 2) * MC_TILE + (k & 3) * 32, 16, 1024, SWZ_128B),
                   make_smem_desc(kb + (k >> 2) * MC_TILE + (k & 3) * 32, 16, 1024, SWZ_128B), id_s, k != 0 ? 1u : 0u);
      }
      for (int term = 0; ok && term < 2; ++term) {
        ok = mbar_wait(full_b, (uint32_t)term, dead, KID_MLSTM, 5);
        if (!ok) break;
        for (int k = 0; k < ks; ++k)
          umma_f16(tmem_o, make_smem_desc(qb + (k >> 2) * MC_TILE + (k & 3) * 32, 16, 1024, SWZ_128B), make_smem_desc(bb + k * 2048, st, 1024, SWZ_128B),
                   id_o, (term | k) != 0 ? 1u : 0u);
        umma_commit(b_free);
      }
      if (ok) {
        umma_commit(o_init);
        ok = mbar_wait(p_ready, 0, dead, KID_MLSTM, 6) && mbar_wait(full_b, 0, dead, KID_MLSTM, 7);
      }
      if (ok) {
        tc_fence_after_sync();
        for (int term = 0; term < 2; ++term)
          for (int k = 0; k < MC / 16; ++k)
            umma_f16(tmem_o, make_smem_desc(pb + (2 * term + (k >> 2)) * MC_TILE + (k & 3) * 32, 16, 1024, SWZ_128B),
                     make_smem_desc(bb + k * 2048, MC_TILE, 1024, SWZ_128B), id_o, 1u);
        umma_commit(o_full);
      }
    }
    __syncwarp();
  } else {
    const int q = warp & 3, t = q * 32 + lane, half = (warp - 2) >> 2;       // TMEM lane quarter, token of the chunk
    const uint32_t lane_off = (uint32_t)(q * 32) << 16;
    const float m0 = p.m0[unit], M = fmaxf(m0, p.lg[unit * 3 * MC + MC + t]), m = p.lg[unit * 3 * MC + 2 * MC + t] + M, w0 = ml_ex2(m0 - M);
    float nq = 0.f;                                          // this thread's part of n_t . q_t
    mbar_wait(full_qk, 0, dead, KID_MLSTM, 8);
    for (int u = half; u < (D >> 3); u += 2) {
      const uint4 raw = *reinterpret_cast<const uint4*>(q_smem + (u >> 3) * MC_TILE + ml_swz(t, u & 7));
      const uint32_t r[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 x = unpack_16<BF16>(r[j]);
        nq = fmaf(x.x, n0[u * 8 + 2 * j], nq);
        nq = fmaf(x.y, n0[u * 8 + 2 * j + 1], nq);
      }
    }
    nq *= w0;
    asm volatile("bar.sync 1, 256;\n" ::: "memory");         // the weighted scores overwrite the queries
    mbar_wait(o_init, 0, dead, KID_MLSTM, 9);
    tc_fence_after_sync();
#pragma unroll 1
    for (int b = half; b < MC / 32; b += 2) {
      uint32_t s[32];
      const bool any = b <= q;                               // (of the warp: blocks above the diagonal are zero)
      if (any) {
        tmem_ld_32x32b_x32(tmem_s + lane_off + b * 32, s);
        tmem_ld_wait();
      }
#pragma unroll
      for (int g = 0; g < 4; ++g) {
        uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
        if (any) {
          float x[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            const int k = b * 32 + g * 8 + j;
            x[j] = k <= t && k < n ? __uint_as_float(s[g * 8 + j]) * ml_ex2(as[k] - M) : 0.f;
            nq += x[j];
          }
          ml_split8<BF16>(x, hi, lo);
        }
        const int at = (b >> 1) * MC_TILE + ml_swz(t, (b & 1) * 4 + g);
        *reinterpret_cast<uint4*>(p_smem + at) = hi;
        *reinterpret_cast<uint4*>(p_smem + 2 * MC_TILE + at) = lo;
      }
    }
#pragma unroll 1
    for (int c0 = half * 32; c0 < V; c0 += 64) {
      uint32_t o[32];
      tmem_ld_32x32b_x32(tmem_o + lane_off + c0, o);
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 32; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * w0);
      tmem_st_32x32b_x32(tmem_o + lane_off + c0, o);
    }
    tmem_st_wait();
    fence_proxy_async_smem();
    tc_fence_before_sync();
    mbar_arrive(p_ready);
    red[half * MC + t] = nq;
    asm volatile("bar.sync 1, 256;\n" ::: "memory");
    nq = (red[t] + red[MC + t]) * p.scale;
    const float f = p.scale / (fmaxf(fabsf(nq), ml_ex2(-m)) + 1e-6f);
    const bool live = t < n;
    const uint16_t* gp = reinterpret_cast<const uint16_t*>(p.proj) + (size_t)(r0 + (live ? t : 0)) * p.ld + p.g_col + (size_t)h * V;
    const uint16_t* wp = reinterpret_cast<const uint16_t*>(p.norm_w) + (size_t)h * V;
    uint16_t* op = reinterpret_cast<uint16_t*>(p.out) + (size_t)(r0 + (live ? t : 0)) * p.ld_out + (size_t)h * V;
    mbar_wait(o_full, 0, dead, KID_MLSTM, 10);
    tc_fence_after_sync();
    float ss = 0.f;
#pragma unroll 1
    for (int c0 = half * 32; c0 < V; c0 += 64) {
      uint32_t o[32];
      tmem_ld_32x32b_x32(tmem_o + lane_off + c0, o);
      tmem_ld_wait();
#pragma unroll
      for (int j = 0; j < 32; ++j)
        if (c0 + j < V) { const float x = __uint_as_float(o[j]) * f; ss = fmaf(x, x, ss); }
    }
    red[2 * MC + half * MC + t] = ss;
    asm volatile("bar.sync 1, 256;\n" ::: "memory");
    ss = red[2 * MC + t] + red[3 * MC + t];
    const float inv = f / sqrtf(ss / (float)V + p.eps);
#pragma unroll 1
    for (int c0 = half * 32; c0 < V; c0 += 64) {
      uint32_t o[32];
      __syncwarp();
      tmem_ld_32x32b_x32(tmem_o + lane_off + c0, o);
      uint4 gv[4];
#pragma unroll
      for (int g = 0; g < 4; ++g)
        if (c0 + 8 * g < V) gv[g] = *reinterpret_cast<const uint4*>(gp + c0 + 8 * g);
      tmem_ld_wait();
      if (!live) continue;
#pragma unroll
      for (int g = 0; g < 4; ++g) {
        if (c0 + 8 * g >= V) break;
        const uint4 wv = *reinterpret_cast<const uint4*>(wp + c0 + 8 * g);
        const uint32_t gr[4] = {gv[g].x, gv[g].y, gv[g].z, gv[g].w}, wr[4] = {wv.x, wv.y, wv.z, wv.w};
        uint32_t y[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 gg = unpack_16<BF16>(gr[j]), ww = unpack_16<BF16>(wr[j]);
          const float a = __uint_as_float(o[8 * g + 2 * j]) * inv * ww.x, b = __uint_as_float(o[8 * g + 2 * j + 1]) * inv * ww.y;
          y[j] = pack_16<BF16>(__fdividef(a, 1.0f + __expf(-gg.x)), __fdividef(b, 1.0f + __expf(-gg.y)));
        }
        *reinterpret_cast<uint4*>(op + c0 + 8 * g) = make_uint4(y[0], y[1], y[2], y[3]);
      }
    }
    if (last_slot >= 0 && half == 0 && t == n - 1) p.state[((size_t)last_slot * p.H + h) * p.st_head + (size_t)D * V + D] = m * ML_LN2;
  }
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_s, tmem_cols);
}

static int mlstm_state_smem(int D, int V) { return ((D + 63) / 64 + 4 * ((V + 127) / 128)) * MC_TILE + (MC + 512 + 8) * 4 + 64 + 1024; }
static int mlstm_out_smem(int D, int V) {
  const int dt = (D + 63) / 64, vt = (V + 63) / 64, Dp = (D + 15) & ~15;
  return (2 * dt > 4 ? 2 * dt : 4) * MC_TILE + vt * (Dp > MC ? Dp : MC) * 128 + (MC + 256 + 4 * MC) * 4 + 64 + 1024;
}
static int mlstm_cols(int n) { int c = 32; while (c < n) c <<= 1; return c; }

}  // namespace fb

using namespace fb;

extern "C" int fb_mlstm_chunk_supported(int D, int V) {
  return D > 0 && V > 0 && D <= 256 && V <= 256 && D % 8 == 0 && V % 8 == 0 && mlstm_state_smem(D, V) <= MC_SMEM_MAX && mlstm_out_smem(D, V) <= MC_SMEM_MAX &&
         ((V + 127) / 128) * ((D + 15) & ~15) <= 512 ? 1 : 0;
}

// See MlstmParams.  items null: token b belongs to request b, state slots[b].  dt: 0 fp16, 1 bf16, 2 fp32.
extern "C" int fb_mlstm_recurrent(const void* proj, long long ld, const float* gates, long long ld_gates, const float* gate_b, const void* norm_w,
                                  float* state, long long st_head, const int* slots, const int* items, void* out, long long ld_out, int B, int H, int D,
                                  int V, int k_col, int v_col, int g_col, float scale, float cap, float eps, int dt, void* stream_) {
  if (B <= 0) return 0;
  if (H <= 0 || D <= 0 || V <= 0 || B > 65535 || D > 8192 || V > 512 || st_head < (long long)D * V + D + 1 || !(cap > 0.f) || dt < 0 || dt > 2 ||
      (slots == nullptr && items == nullptr))
    return -1;
  MlstmParams p = {};
  p.proj = proj; p.ld = ld; p.gates = gates; p.ld_gates = ld_gates; p.gate_b = gate_b; p.norm_w = norm_w; p.state = state; p.st_head = st_head;
  p.slots = slots; p.items = items; p.out = out; p.ld_out = ld_out; p.H = H; p.D = D; p.V = V; p.k_col = k_col; p.v_col = v_col; p.g_col = g_col;
  p.scale = scale; p.cap = cap; p.eps = eps;
  const int cgs = (V + 31) / 32;
  int R = 0, rgs = 1;
  for (int warps = 8; warps <= 16 && R == 0; warps *= 2)       // 256 threads where the state fits their registers, else 512
    for (int r = 16; r <= 64; r *= 2) {
      const int g = (D + r - 1) / r;
      if (cgs * g <= warps) { R = r; rgs = g; break; }
    }
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  if (R == 0) {
    rgs = 16 / cgs;
    if (rgs > D) rgs = D;
  }
  const int threads = cgs * rgs * 32;
  const int rows = R > 0 ? R : (D + rgs - 1) / rgs;
  const size_t smem = (size_t)(3 * ((rows * rgs + 3) & ~3) + rgs * 32 * cgs + 32) * 4;
  if (smem > 200 * 1024) return -1;
#define GO2(DT, RR)                                                                                                                          \
  {                                                                                                                                          \
    static DeviceOnce cfg;                                                                                                                   \
    if (cfg.need()) cudaFuncSetAttribute(mlstm_recurrent_kernel<DT, RR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);            \
    launch_k(mlstm_recurrent_kernel<DT, RR>, dim3(H, B), dim3(threads), smem, stream, 0, p, rgs);                                            \
  }
#define GO(DT) { if (R == 16) GO2(DT, 16) else if (R == 32) GO2(DT, 32) else if (R == 64) GO2(DT, 64) else GO2(DT, 0) }
  if (dt == 0) GO(0) else if (dt == 1) GO(1) else GO(2)
#undef GO
#undef GO2
  return (int)cudaGetLastError();
}

// Chunked form over the heads [h0, h0 + Hn): chunks / reqs as in MlstmParams; scratch, with units = n_chunks * Hn: inc [units * D * V], ninc and
// n0 [units * D], lg [units * 384], m0 [units] floats, s0 [units * 2 * Dp * V] 16-bit values (zero in the rows D .. Dp - 1, Dp = D rounded
// up to 16).  16-bit projections [T, ld], widths as fb_mlstm_chunk_supported says.
extern "C" int fb_mlstm_chunked(const void* proj, long long ld, int T, const float* gates, long long ld_gates, const float* gate_b, const void* norm_w,
                                float* state, long long st_head, const int* chunks, int n_chunks, const int* reqs, int n_reqs, float* inc, float* ninc,
                                float* lg, float* m0, float* n0, void* s0, void* out, long long ld_out, int H, int h0, int Hn, int D, int V, int k_col,
                                int v_col, int g_col, float scale, float cap, float eps, int dt, void* stream_) {
  if (n_chunks <= 0 || n_reqs <= 0) return 0;
  if (!fb_mlstm_chunk_supported(D, V) || T <= 0 || H <= 0 || h0 < 0 || Hn <= 0 || h0 + Hn > H || Hn > 65535 || n_reqs > 65535 || ld % 8 != 0 || k_col % 8 != 0 ||
      v_col % 8 != 0 || g_col % 8 != 0 || ld_out % 8 != 0 || st_head % 2 != 0 || st_head < (long long)D * V + D + 1 || !(cap > 0.f) ||
      (reinterpret_cast<uintptr_t>(proj) & 15) || (reinterpret_cast<uintptr_t>(out) & 15) || (dt != 0 && dt != 1))
    return -1;
  MlstmParams p = {};
  p.proj = proj; p.ld = ld; p.gates = gates; p.ld_gates = ld_gates; p.gate_b = gate_b; p.norm_w = norm_w; p.state = state; p.st_head = st_head;
  p.chunks = chunks; p.n_chunks = n_chunks; p.reqs = reqs; p.inc = inc; p.ninc = ninc; p.lg = lg; p.m0 = m0; p.n0 = n0; p.s0 = (uint16_t*)s0;
  p.out = out; p.ld_out = ld_out; p.H = H; p.h0 = h0; p.Hn = Hn; p.D = D; p.V = V; p.k_col = k_col; p.v_col = v_col; p.g_col = g_col;
  p.scale = scale; p.cap = cap; p.eps = eps; p.Dp = (D + 15) & ~15;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  const uint16_t* base = reinterpret_cast<const uint16_t*>(proj);
  CUtensorMap tmQ, tmK, tmV, tmS;
  if (!make_tmap_3d(&tmQ, base, D, H, T, D, ld, 64, MC) || !make_tmap_3d(&tmK, base + k_col, D, H, T, D, ld, 64, MC) ||
      !make_tmap_3d(&tmV, base + v_col, V, H, T, V, ld, 64, MC) ||
      !make_tmap_2d(&tmS, s0, (uint64_t)n_chunks * Hn * 2 * p.Dp, V, V, p.Dp, 64, 2, 3))
    return -2;
  const int state_cols = mlstm_cols(((V + 127) / 128) * p.Dp), out_cols = mlstm_cols(MC + (V + 63) / 64 * 64);
  const int sm_state = mlstm_state_smem(D, V), sm_out = mlstm_out_smem(D, V);
  const dim3 grid(n_chunks, Hn), scan((D * V + D + 255) / 256, Hn, n_reqs);
#define FB_ML(BF)                                                                                                             \
  {                                                                                                                           \
    static DeviceOnce cfg;                                                                                                    \
    if (cfg.need()) {                                                                                                         \
      cudaFuncSetAttribute(mlstm_chunk_state_kernel<BF>, cudaFuncAttributeMaxDynamicSharedMemorySize, MC_SMEM_MAX);            \
      cudaFuncSetAttribute(mlstm_chunk_out_kernel<BF>, cudaFuncAttributeMaxDynamicSharedMemorySize, MC_SMEM_MAX);              \
    }                                                                                                                         \
    launch_k(mlstm_chunk_state_kernel<BF>, grid, dim3(MC_STATE_THREADS), sm_state, stream, 0, tmK, p, state_cols);            \
    launch_k(mlstm_chunk_scan_kernel<BF>, scan, dim3(128), 0, stream, 0, p);                                                  \
    launch_k(mlstm_chunk_out_kernel<BF>, grid, dim3(MC_OUT_THREADS), sm_out, stream, 0, tmQ, tmK, tmV, tmS, p, out_cols);                \
  }
  if (dt == 1) FB_ML(true) else FB_ML(false)
#undef FB_ML
  return (int)cudaGetLastError();
}
