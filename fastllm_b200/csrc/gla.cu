// Gated linear attention for sm_100a: per head a [D, V] fp32 state whose key channels decay at their own data-dependent rate,
//     S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,   alpha_t = sigmoid(W_a2 a_t + b)^(1 / tau),
// then RMS norm of every head's output and * silu(gate).  q, k, v, gate and a_t are columns of one merged projection row.
//
//  * gla_recurrent_kernel: one CTA per (head, request) walks the request's tokens with the state in registers; a thread owns R rows of
//    one state column, so the state is read once and written once per step.  Any widths, fp32 included.
//  * the chunked form for prompts, 64 tokens per chunk, every chunk and head in parallel except for the scan:
//      gla_chunk_state   U_c = sum_t (k_t exp(b_C - b_t)) v_t^T         (the state's increment over the chunk; b: running log-decay)
//      gla_chunk_scan    S_c = exp(b_C) S_(c-1) + U_c                   (leaves S_(c-1) in place of U_c, the last one in the slot)
//      gla_chunk_out     o_t = S_(c-1)^T (q_t exp(b_t)) + sum_(s <= t) A_ts v_s,  A_ts = sum_d q_td k_sd exp(b_td - b_sd)
//    Exponents are differences forwards in time and never positive: across blocks of 16 tokens the difference is split at the later
//    block's first token, inside a block it is taken pair by pair.  Products run on tf32 operands (q, k and the state carry ten
//    fraction bits beyond which bf16 inputs have nothing left but the decay factors) with fp32 accumulation; the state stays fp32.
//
// Compiled without fast-math: log-decays, norms and gates of the recurrence are the correctly rounded fp32 ones.
#include "ptx.cuh"
#include "launch.h"

FB_DEFINE_ERROR_API(gla)

namespace fb {

template <int DT> struct GAct;
template <> struct GAct<0> { typedef uint16_t T; static __device__ __forceinline__ float ld(uint16_t v) { return __half2float(__ushort_as_half(v)); }
                             static __device__ __forceinline__ uint16_t st(float v) { return __half_as_ushort(__float2half_rn(v)); } };
template <> struct GAct<1> { typedef uint16_t T; static __device__ __forceinline__ float ld(uint16_t v) { return __bfloat162float(__ushort_as_bfloat16(v)); }
                             static __device__ __forceinline__ uint16_t st(float v) { return __bfloat16_as_ushort(__float2bfloat16_rn(v)); } };
template <> struct GAct<2> { typedef float T; static __device__ __forceinline__ float ld(float v) { return v; } static __device__ __forceinline__ float st(float v) { return v; } };

struct GlaParams {
  const void* proj; long long ld;          // [T, ld] rows: queries from column 0, then keys, values, gate, decay rank at *_col
  const void* a2; const void* a2_b;        // [H * D, rank], [H * D]
  const void* norm_w;                      // [V]
  float* state;                            // [slots, H, D, V]
  void* out; long long ld_out;             // [T, H * V]
  int H, D, V, rank, k_col, v_col, g_col, a_col;
  float scale, inv_tau, eps;
  // recurrent form
  const int* slots; const int* cu;         // [B]; cu [B + 1] token offsets (null: token b belongs to request b)
  // chunked form
  const int* chunks; const int* reqs;      // [n_chunks][2] = (first row, rows); [n_reqs][3] = (first chunk, chunks, slot)
  float* inc; float* dec;                  // [n_chunks, Hn, D, V], [n_chunks, Hn, D]
  int n_chunks, h0, Hn;
};

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------------------------------------------
// recurrent form
// ------------------------------------------------------------------------------------------------
// Threads: ceil(V / 32) column groups x row groups of R rows; R = 0: the state stays in memory (widths beyond the register forms).
template <int DT, int R>
__global__ void __launch_bounds__(512) gla_recurrent_kernel(const GlaParams p, int row_groups) {
  typedef typename GAct<DT>::T T;
  extern __shared__ float sm[];
  const int D = p.D, V = p.V, tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31;
  const int cgs = (V + 31) >> 5;
  const int rows = R > 0 ? R : (D + row_groups - 1) / row_groups, Dp = (rows * row_groups + 3) & ~3;
  float* qs = sm;                    // [Dp] (zero beyond D)
  float* ks = qs + Dp;
  float* al = ks + Dp;
  float* part = al + Dp;             // [row_groups][32 * cgs]
  float* red = part + row_groups * 32 * cgs;     // [16]
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y;
  const int t0 = p.cu != nullptr ? p.cu[b] : b, t1 = p.cu != nullptr ? p.cu[b + 1] : b + 1;
  if (t1 <= t0) return;
  const int cg = warp % cgs, rg = warp / cgs, j = cg * 32 + lane;
  const bool col = j < V;
  float* S = p.state + ((size_t)p.slots[b] * p.H + h) * D * V;
  const int r0 = rg * rows, rn = min(rows, D - r0);
  for (int d = D + tid; d < Dp; d += nt) { qs[d] = 0.f; ks[d] = 0.f; al[d] = 0.f; }
  float s[R > 0 ? R : 1];
  if (R > 0) {
#pragma unroll
    for (int i = 0; i < R; ++i) s[i] = (col && i < rn) ? S[(size_t)(r0 + i) * V + j] : 0.f;
  }
  const T* a2 = reinterpret_cast<const T*>(p.a2) + (size_t)h * D * p.rank;
  const T* ab = reinterpret_cast<const T*>(p.a2_b) + (size_t)h * D;
  const T* nw = reinterpret_cast<const T*>(p.norm_w);
  for (int t = t0; t < t1; ++t) {
    const T* row = reinterpret_cast<const T*>(p.proj) + (size_t)t * p.ld;
    const T* ar = row + p.a_col;
    for (int d = tid; d < D; d += nt) {
      qs[d] = GAct<DT>::ld(row[h * D + d]) * p.scale;
      ks[d] = GAct<DT>::ld(row[p.k_col + h * D + d]);
      float z = GAct<DT>::ld(ab[d]);
      const T* w = a2 + (size_t)d * p.rank;
#pragma unroll 4
      for (int r = 0; r < p.rank; ++r) z = fmaf(GAct<DT>::ld(w[r]), GAct<DT>::ld(ar[r]), z);
      al[d] = expf(log_sigmoid(z) * p.inv_tau);
    }
    const float v = col ? GAct<DT>::ld(row[p.v_col + h * V + j]) : 0.f;
    __syncthreads();
    float o = 0.f;
    if (R > 0) {
      const float4 *k4 = reinterpret_cast<const float4*>(ks + r0), *a4 = reinterpret_cast<const float4*>(al + r0), *q4 = reinterpret_cast<const float4*>(qs + r0);
#pragma unroll
      for (int i = 0; i < R / 4; ++i) {
        const float4 kk = k4[i], aa = a4[i], qq = q4[i];
        s[4 * i] = fmaf(s[4 * i], aa.x, kk.x * v); s[4 * i + 1] = fmaf(s[4 * i + 1], aa.y, kk.y * v);
        s[4 * i + 2] = fmaf(s[4 * i + 2], aa.z, kk.z * v); s[4 * i + 3] = fmaf(s[4 * i + 3], aa.w, kk.w * v);
        o = fmaf(s[4 * i], qq.x, o); o = fmaf(s[4 * i + 1], qq.y, o); o = fmaf(s[4 * i + 2], qq.z, o); o = fmaf(s[4 * i + 3], qq.w, o);
        if ((i & 3) == 3) asm volatile("" ::: "memory");       // keeps the reads of a few rows in flight, not of all of them
      }
    } else if (col) {
      for (int i = 0; i < rn; ++i) {
        float* sp = S + (size_t)(r0 + i) * V + j;
        const float n = fmaf(*sp, al[r0 + i], ks[r0 + i] * v);
        *sp = n;
        o = fmaf(n, qs[r0 + i], o);
      }
    }
    part[rg * 32 * cgs + j] = o;
    __syncthreads();
    // output of the head: sum over the row groups, norm over V, gate
    float ss = 0.f;
    for (int i = tid; i < V; i += nt) {
      float x = part[i];
      for (int g = 1; g < row_groups; ++g) x += part[g * 32 * cgs + i];
      part[i] = x;
      ss += x * x;
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.f;
    for (int w = 0; w < (nt >> 5); ++w) ss += red[w];
    const float inv = 1.0f / sqrtf(ss / (float)V + p.eps);
    for (int i = tid; i < V; i += nt) {
      const float g = GAct<DT>::ld(row[p.g_col + h * V + i]);
      const float y = part[i] * inv * GAct<DT>::ld(nw[i]);
      reinterpret_cast<T*>(p.out)[(size_t)t * p.ld_out + (size_t)h * V + i] = GAct<DT>::st(y * (g / (1.0f + expf(-g))));
    }
    __syncthreads();                     // part / red / qs are rewritten by the next token
  }
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
constexpr int GC = 64;                         // tokens per chunk
constexpr int GC_THREADS = 256;
constexpr int GC_MAX_RANK = 64;

__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float to_tf32(float x) { uint32_t y; asm("cvt.rna.tf32.f32 %0, %1;\n" : "=r"(y) : "f"(x)); return __uint_as_float(y); }
__device__ __forceinline__ void mma_tf32(float* c, const float* a, float b0, float b1) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(__float_as_uint(a[0])), "r"(__float_as_uint(a[1])), "r"(__float_as_uint(a[2])), "r"(__float_as_uint(a[3])),
                 "r"(__float_as_uint(b0)), "r"(__float_as_uint(b1)));
}
// row strides that keep the fragment reads free of bank conflicts
__host__ __device__ constexpr int gc_ld_state(int D) { return (D + 31) / 32 * 32 + 8; }       // fp32, a fragment's rows run along d
__host__ __device__ constexpr int gc_ld_out(int D) { return (D + 31) / 32 * 32 + 4; }         // fp32, rows run along the tokens
__host__ __device__ constexpr int gc_ld_v(int V) { return (V + 63) / 64 * 64 + 16; }          // 16-bit values
__host__ __device__ constexpr int gc_ld_qk(int D) { return (D + 63) / 64 * 64 + 8; }          // 16-bit queries / keys
constexpr int GC_LD_A = GC + 4;

// rows [row0, row0 + n) of `width` 16-bit columns into shared memory, zero rows behind them
__device__ __forceinline__ void gc_load(const uint16_t* src, long long ld, int n, int width, uint16_t* dst, int ld_dst) {
  const int vecs = width >> 3;
  for (int i = threadIdx.x; i < GC * vecs; i += GC_THREADS) {
    const int t = i / vecs, c = (i - t * vecs) << 3;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (t < n) v = *reinterpret_cast<const uint4*>(src + (size_t)t * ld + c);
    *reinterpret_cast<uint4*>(dst + (size_t)t * ld_dst + c) = v;
  }
}

// Running log2-decay of the chunk's tokens, bc[t][d] (rows beyond n decay by nothing).  a1: scratch [GC][rank rounded up to 16].
// Ends with the chunk's totals known to the thread's column: every thread returns bc[GC - 1][d] of the column it handled.
template <int DT>
__device__ __forceinline__ void gc_decay(const GlaParams& p, const uint16_t* row0, int n, int h, float* bc, int ldb, float* a1, float* tot) {
  const int D = p.D, rp = (p.rank + 15) & ~15;
  for (int i = threadIdx.x; i < GC * rp; i += GC_THREADS) {
    const int t = i / rp, r = i - t * rp;
    a1[i] = (t < n && r < p.rank) ? GAct<DT>::ld(row0[(size_t)t * p.ld + p.a_col + r]) : 0.f;
  }
  __syncthreads();
  const int parts = D <= 64 ? 4 : D <= 128 ? 2 : 1, tp = GC / parts;
  const int wd = GC_THREADS / parts;                      // columns per part, at least D
  const int part = threadIdx.x / wd, d = threadIdx.x - part * wd;
  const uint16_t* a2 = reinterpret_cast<const uint16_t*>(p.a2) + ((size_t)h * D + (d < D ? d : 0)) * p.rank;
  if (d < D) {
    const float bias = GAct<DT>::ld(reinterpret_cast<const uint16_t*>(p.a2_b)[h * D + d]);
    for (int r0 = 0; r0 < rp; r0 += 16) {
      float w[16];
#pragma unroll
      for (int r = 0; r < 16; ++r) w[r] = r0 + r < p.rank ? GAct<DT>::ld(a2[r0 + r]) : 0.f;
      float run = 0.f;
      for (int t = part * tp; t < (part + 1) * tp; ++t) {
        float z = r0 == 0 ? bias : bc[t * ldb + d];
        const float4* ap = reinterpret_cast<const float4*>(a1 + t * rp + r0);
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          const float4 a = ap[r];
          z = fmaf(w[4 * r], a.x, z); z = fmaf(w[4 * r + 1], a.y, z); z = fmaf(w[4 * r + 2], a.z, z); z = fmaf(w[4 * r + 3], a.w, z);
        }
        if (r0 + 16 >= rp) {
          if (t < n) run += log_sigmoid(z) * p.inv_tau * 1.4426950408889634f;
          z = run;
        }
        bc[t * ldb + d] = z;
      }
      tot[part * wd + d] = run;
    }
  }
  __syncthreads();
  if (d < D && part > 0) {
    float off = 0.f;
    for (int q = 0; q < part; ++q) off += tot[q * wd + d];
    for (int t = part * tp; t < (part + 1) * tp; ++t) bc[t * ldb + d] += off;
  }
  __syncthreads();
}

template <int DT>
__global__ void __launch_bounds__(GC_THREADS) gla_chunk_state_kernel(const GlaParams p) {
  extern __shared__ float sm[];
  const int D = p.D, V = p.V, ldb = gc_ld_state(D), ldv = gc_ld_v(V), rp = (p.rank + 15) & ~15;
  float* kt = sm;                                                     // [GC][ldb] log-decays, then decayed keys
  float* a1 = kt + GC * ldb;                                          // [GC][rp]
  float* tot = a1 + GC * rp;                                          // [GC_THREADS]
  uint16_t* vs = reinterpret_cast<uint16_t*>(tot + GC_THREADS);       // [GC][ldv]
  const int c = blockIdx.x, hl = blockIdx.y, h = p.h0 + hl;
  const int r0 = p.chunks[2 * c], n = p.chunks[2 * c + 1];
  const uint16_t* row0 = reinterpret_cast<const uint16_t*>(p.proj) + (size_t)r0 * p.ld;
  gc_load(row0 + p.v_col + h * V, p.ld, n, V, vs, ldv);
  gc_decay<DT>(p, row0, n, h, kt, ldb, a1, tot);
  const uint16_t* kp = row0 + p.k_col + h * D;
  const size_t unit = (size_t)c * p.Hn + hl;
  const int parts = D <= 64 ? 4 : D <= 128 ? 2 : 1, tp = GC / parts, wd = GC_THREADS / parts;
  const int part = threadIdx.x / wd, d = threadIdx.x - part * wd;
  float last = 0.f;
  if (d < D) last = kt[(GC - 1) * ldb + d];
  __syncthreads();                                                    // (the last row is overwritten below by another part)
  if (d < D) {
    if (part == 0) p.dec[unit * D + d] = ex2(last);
    for (int t = part * tp; t < (part + 1) * tp; ++t) {
      const float k = t < n ? GAct<DT>::ld(kp[(size_t)t * p.ld + d]) : 0.f;
      kt[t * ldb + d] = to_tf32(k * ex2(last - kt[t * ldb + d]));
    }
  }
  __syncthreads();
  // U[d][v] = sum_t K~[t][d] V[t][v]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  const int mbs = (D + 15) >> 4, nts = V >> 3, ngs = (nts + 7) >> 3;
  float* U = p.inc + unit * D * V;
  for (int u = warp; u < mbs * ngs; u += GC_THREADS / 32) {
    const int mb = u % mbs, nt0 = (u / mbs) * 8, cnt = min(8, nts - nt0);
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) { acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f; }
#pragma unroll 2
    for (int k0 = 0; k0 < GC; k0 += 8) {
      const float* ap = kt + (k0 + q) * ldb + mb * 16 + g;
      const float a[4] = {ap[0], ap[8], ap[4 * ldb], ap[4 * ldb + 8]};
      const uint16_t* bp = vs + (k0 + q) * ldv + nt0 * 8 + g;
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i < cnt) mma_tf32(acc[i], a, GAct<DT>::ld(bp[i * 8]), GAct<DT>::ld(bp[4 * ldv + i * 8]));
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (i >= cnt) break;
      const int v = (nt0 + i) * 8 + 2 * q, d0 = mb * 16 + g;
      if (d0 < D) *reinterpret_cast<float2*>(U + (size_t)d0 * V + v) = make_float2(acc[i][0], acc[i][1]);
      if (d0 + 8 < D) *reinterpret_cast<float2*>(U + (size_t)(d0 + 8) * V + v) = make_float2(acc[i][2], acc[i][3]);
    }
  }
}

// one thread per four state elements of a (request, head); reads run ahead of the dependent chain
__global__ void __launch_bounds__(256) gla_chunk_scan_kernel(const GlaParams p) {
  const int D = p.D, V = p.V, hl = blockIdx.y;
  const int e = (blockIdx.x * 256 + threadIdx.x) * 4;
  if (e >= D * V) return;
  const int c0 = p.reqs[3 * blockIdx.z], n = p.reqs[3 * blockIdx.z + 1], slot = p.reqs[3 * blockIdx.z + 2];
  const int d = e / V;
  float4* st = reinterpret_cast<float4*>(p.state + ((size_t)slot * p.H + p.h0 + hl) * D * V + e);
  float4 s = *st;
  const size_t su = (size_t)p.Hn * D * V, sd = (size_t)p.Hn * D;
  float* U = p.inc + ((size_t)c0 * p.Hn + hl) * D * V + e;
  const float* dc = p.dec + ((size_t)c0 * p.Hn + hl) * D + d;
  constexpr int A = 8;
  for (int c = 0; c < n; c += A) {
    float4 u[A];
    float f[A];
#pragma unroll
    for (int i = 0; i < A; ++i)
      if (c + i < n) { u[i] = *reinterpret_cast<const float4*>(U + (size_t)(c + i) * su); f[i] = dc[(size_t)(c + i) * sd]; }
#pragma unroll
    for (int i = 0; i < A; ++i) {
      if (c + i >= n) break;
      *reinterpret_cast<float4*>(U + (size_t)(c + i) * su) = s;
      s.x = fmaf(s.x, f[i], u[i].x); s.y = fmaf(s.y, f[i], u[i].y); s.z = fmaf(s.z, f[i], u[i].z); s.w = fmaf(s.w, f[i], u[i].w);
    }
  }
  *st = s;
}

// NTW: 8-column output tiles per warp, ceil(V / 64)
template <int DT, int NTW>
__global__ void __launch_bounds__(GC_THREADS) gla_chunk_out_kernel(const GlaParams p) {
  extern __shared__ float sm[];
  const int D = p.D, V = p.V, ldb = gc_ld_out(D), ldq = gc_ld_qk(D), ldv = gc_ld_v(V);
  float* bc = sm;                                                     // [GC][ldb] log-decays, then decayed queries
  float* At = bc + GC * ldb;                                          // [GC][GC_LD_A]; before that the decay's scratch
  float* tot = At + GC * GC_LD_A;                                     // [GC_THREADS]
  float* red = tot + GC_THREADS;                                      // [8][GC]
  uint16_t* qs = reinterpret_cast<uint16_t*>(red + 8 * GC);           // [GC][ldq]
  uint16_t* ks = qs + GC * ldq;
  uint16_t* vs = ks + GC * ldq;                                       // [GC][ldv]
  const int c = blockIdx.x, hl = blockIdx.y, h = p.h0 + hl;
  const int r0 = p.chunks[2 * c], n = p.chunks[2 * c + 1];
  const uint16_t* row0 = reinterpret_cast<const uint16_t*>(p.proj) + (size_t)r0 * p.ld;
  gc_load(row0 + h * D, p.ld, n, D, qs, ldq);
  gc_load(row0 + p.k_col + h * D, p.ld, n, D, ks, ldq);
  gc_load(row0 + p.v_col + h * V, p.ld, n, V, vs, ldv);
  gc_decay<DT>(p, row0, n, h, bc, ldb, At, tot);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  for (int i = threadIdx.x; i < GC * GC_LD_A; i += GC_THREADS) At[i] = 0.f;
  __syncthreads();
  // A between blocks of 16 tokens (i > j): the exponent is split at the token before block i
  if (warp < 6) {
    const int i = warp < 1 ? 1 : warp < 3 ? 2 : 3, j = warp - (i * (i - 1)) / 2;
    const float* ref = bc + (16 * i - 1) * ldb;
    float acc[2][4] = {};
    const float* bt = bc + (16 * i + g) * ldb;
    const uint16_t* qt = qs + (16 * i + g) * ldq;
    const float* bs = bc + (16 * j + g) * ldb;
    const uint16_t* ksr = ks + (16 * j + g) * ldq;
#pragma unroll 2
    for (int k0 = 0; k0 < D; k0 += 8) {
      const int da = k0 + q, db = da + 4;
      const float ra = ref[da], rb = ref[db];
      const float a[4] = {to_tf32(GAct<DT>::ld(qt[da]) * ex2(bt[da] - ra)), to_tf32(GAct<DT>::ld(qt[8 * ldq + da]) * ex2(bt[8 * ldb + da] - ra)),
                          to_tf32(GAct<DT>::ld(qt[db]) * ex2(bt[db] - rb)), to_tf32(GAct<DT>::ld(qt[8 * ldq + db]) * ex2(bt[8 * ldb + db] - rb))};
#pragma unroll
      for (int m = 0; m < 2; ++m)
        mma_tf32(acc[m], a, to_tf32(GAct<DT>::ld(ksr[m * 8 * ldq + da]) * ex2(ra - bs[m * 8 * ldb + da])),
                 to_tf32(GAct<DT>::ld(ksr[m * 8 * ldq + db]) * ex2(rb - bs[m * 8 * ldb + db])));
    }
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      float* o = At + (16 * i + g) * GC_LD_A + 16 * j + m * 8 + 2 * q;
      o[0] = to_tf32(acc[m][0] * p.scale); o[1] = to_tf32(acc[m][1] * p.scale);
      o[8 * GC_LD_A] = to_tf32(acc[m][2] * p.scale); o[8 * GC_LD_A + 1] = to_tf32(acc[m][3] * p.scale);
    }
  }
  // A inside a block: pair by pair, a warp takes rows w and 15 - w of every block (17 pairs each)
  for (int rr = 0; rr < 8; ++rr) {
    const int blk = rr >> 1, t = 16 * blk + ((rr & 1) ? 15 - warp : warp);
    if (t >= n) continue;
    float bt[8], qt[8];
#pragma unroll
    for (int m = 0; m < 8; ++m) {
      const int d = lane + 32 * m;
      bt[m] = d < D ? bc[t * ldb + d] : 0.f;
      qt[m] = d < D ? GAct<DT>::ld(qs[t * ldq + d]) : 0.f;
    }
    for (int s = 16 * blk; s <= t; ++s) {
      float x = 0.f;
#pragma unroll
      for (int m = 0; m < 8; ++m) {
        const int d = lane + 32 * m;
        if (d < D) x = fmaf(qt[m] * GAct<DT>::ld(ks[s * ldq + d]), ex2(bt[m] - bc[s * ldb + d]), x);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
      if (lane == 0) At[t * GC_LD_A + s] = to_tf32(x * p.scale);
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < GC * (D >> 2); i += GC_THREADS) {     // decayed queries, in place
    const int t = i / (D >> 2), d = (i - t * (D >> 2)) << 2;
    float4 b = *reinterpret_cast<float4*>(bc + t * ldb + d);
    const uint16_t* qp = qs + t * ldq + d;
    b.x = to_tf32(GAct<DT>::ld(qp[0]) * p.scale * ex2(b.x)); b.y = to_tf32(GAct<DT>::ld(qp[1]) * p.scale * ex2(b.y));
    b.z = to_tf32(GAct<DT>::ld(qp[2]) * p.scale * ex2(b.z)); b.w = to_tf32(GAct<DT>::ld(qp[3]) * p.scale * ex2(b.w));
    *reinterpret_cast<float4*>(bc + t * ldb + d) = b;
  }
  __syncthreads();
  // O = Q~ S + A V: a warp owns NTW column tiles for all 64 rows, so the state is read once
  const float* S = p.inc + ((size_t)c * p.Hn + hl) * D * V;
  float acc[4][NTW][4];
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int i = 0; i < NTW; ++i) { acc[m][i][0] = acc[m][i][1] = acc[m][i][2] = acc[m][i][3] = 0.f; }
  const int v0 = warp * NTW * 8;
#pragma unroll 4
  for (int k0 = 0; k0 < D; k0 += 8) {
    float b0[NTW], b1[NTW];
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
      const int v = v0 + i * 8 + g;
      b0[i] = v < V ? S[(size_t)(k0 + q) * V + v] : 0.f;
      b1[i] = v < V ? S[(size_t)(k0 + q + 4) * V + v] : 0.f;
    }
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      const float* ap = bc + (16 * m + g) * ldb + k0 + q;
      const float a[4] = {ap[0], ap[8 * ldb], ap[4], ap[8 * ldb + 4]};
#pragma unroll
      for (int i = 0; i < NTW; ++i) mma_tf32(acc[m][i], a, to_tf32(b0[i]), to_tf32(b1[i]));
    }
  }
#pragma unroll 2
  for (int k0 = 0; k0 < GC; k0 += 8) {
    float b0[NTW], b1[NTW];
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
      const int v = v0 + i * 8 + g;
      b0[i] = v < V ? GAct<DT>::ld(vs[(k0 + q) * ldv + v]) : 0.f;
      b1[i] = v < V ? GAct<DT>::ld(vs[(k0 + q + 4) * ldv + v]) : 0.f;
    }
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      if (k0 >= 16 * (m + 1)) continue;                               // above the diagonal
      const float* ap = At + (16 * m + g) * GC_LD_A + k0 + q;
      const float a[4] = {ap[0], ap[8 * GC_LD_A], ap[4], ap[8 * GC_LD_A + 4]};
#pragma unroll
      for (int i = 0; i < NTW; ++i) mma_tf32(acc[m][i], a, b0[i], b1[i]);
    }
  }
  // norm over the head's V columns, weight, gate
#pragma unroll
  for (int m = 0; m < 4; ++m) {
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
      s0 += acc[m][i][0] * acc[m][i][0] + acc[m][i][1] * acc[m][i][1];
      s1 += acc[m][i][2] * acc[m][i][2] + acc[m][i][3] * acc[m][i][3];
    }
    s0 += __shfl_xor_sync(0xffffffffu, s0, 1); s0 += __shfl_xor_sync(0xffffffffu, s0, 2);
    s1 += __shfl_xor_sync(0xffffffffu, s1, 1); s1 += __shfl_xor_sync(0xffffffffu, s1, 2);
    if (q == 0) { red[warp * GC + 16 * m + g] = s0; red[warp * GC + 16 * m + 8 + g] = s1; }
  }
  __syncthreads();
  const uint16_t* nw = reinterpret_cast<const uint16_t*>(p.norm_w);
#pragma unroll
  for (int m = 0; m < 4; ++m) {
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int t = 16 * m + 8 * hf + g;
      if (t >= n) continue;
      float ss = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) ss += red[w * GC + t];
      const float inv = 1.0f / sqrtf(ss / (float)V + p.eps);
      const uint16_t* gp = row0 + (size_t)t * p.ld + p.g_col + h * V;
      uint16_t* op = reinterpret_cast<uint16_t*>(p.out) + (size_t)(r0 + t) * p.ld_out + (size_t)h * V;
#pragma unroll
      for (int i = 0; i < NTW; ++i) {
        const int v = v0 + i * 8 + 2 * q;
        if (v >= V) continue;
        const float2 gv = unpack_16<DT == 1>(*reinterpret_cast<const uint32_t*>(gp + v));
        const float2 wv = unpack_16<DT == 1>(*reinterpret_cast<const uint32_t*>(nw + v));
        const float y0 = acc[m][i][2 * hf] * inv * wv.x * (gv.x / (1.0f + __expf(-gv.x)));
        const float y1 = acc[m][i][2 * hf + 1] * inv * wv.y * (gv.y / (1.0f + __expf(-gv.y)));
        *reinterpret_cast<uint32_t*>(op + v) = pack_16<DT == 1>(y0, y1);
      }
    }
  }
}

}  // namespace fb

using namespace fb;

// See GlaParams.  cu null: one token per request (decode).  dt: 0 fp16, 1 bf16, 2 fp32.
extern "C" int fb_gla_recurrent(const void* proj, long long ld, const void* a2, const void* a2_b, const void* norm_w, float* state,
                                const int* slots, const int* cu, void* out, long long ld_out, int B, int H, int D, int V, int rank, int k_col,
                                int v_col, int g_col, int a_col, float scale, float inv_tau, float eps, int dt, void* stream_) {
  if (B <= 0) return 0;
  if (H <= 0 || D <= 0 || V <= 0 || rank <= 0 || B > 65535 || D > 8192 || V > 8192 || dt < 0 || dt > 2) return -1;
  GlaParams p = {};
  p.proj = proj; p.ld = ld; p.a2 = a2; p.a2_b = a2_b; p.norm_w = norm_w; p.state = state; p.slots = slots; p.cu = cu; p.out = out; p.ld_out = ld_out;
  p.H = H; p.D = D; p.V = V; p.rank = rank; p.k_col = k_col; p.v_col = v_col; p.g_col = g_col; p.a_col = a_col;
  p.scale = scale; p.inv_tau = inv_tau; p.eps = eps;
  const int cgs = (V + 31) / 32;
  int R = 0, rgs = 1;
  for (int r = 16; r <= 64; r *= 2) {
    const int g = (D + r - 1) / r;
    if (cgs * g <= (r == 16 ? 8 : 16)) { R = r; rgs = g; break; }
  }
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  if (R == 0) {
    if (cgs > 16) return -1;                   // heads wider than 512 columns
    rgs = 16 / cgs;
    if (rgs > D) rgs = D;
  }
  const int threads = cgs * rgs * 32;
  const int rows = R > 0 ? R : (D + rgs - 1) / rgs;
  const size_t smem = (size_t)(3 * ((rows * rgs + 3) & ~3) + rgs * 32 * cgs + 16) * 4;
  if (smem > 200 * 1024) return -1;
#define GO2(DT, RR)                                                                                                                          \
  {                                                                                                                                          \
    static DeviceOnce cfg;                                                                                                                   \
    if (cfg.need()) cudaFuncSetAttribute(gla_recurrent_kernel<DT, RR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);              \
    launch_k(gla_recurrent_kernel<DT, RR>, dim3(H, B), dim3(threads), smem, stream, 0, p, rgs);                                              \
  }
#define GO(DT) { if (R == 16) GO2(DT, 16) else if (R == 32) GO2(DT, 32) else if (R == 64) GO2(DT, 64) else GO2(DT, 0) }
  if (dt == 0) GO(0) else if (dt == 1) GO(1) else GO(2)
#undef GO
#undef GO2
  return (int)cudaGetLastError();
}

// Chunked form over the heads [h0, h0 + Hn): chunks / reqs as in GlaParams, scratch inc [n_chunks * Hn * D * V], dec [n_chunks * Hn * D]
// floats.  16-bit projections, D and V multiples of 8 up to 256, rank up to 64.
extern "C" int fb_gla_chunked(const void* proj, long long ld, const void* a2, const void* a2_b, const void* norm_w, float* state,
                              const int* chunks, int n_chunks, const int* reqs, int n_reqs, float* inc, float* dec, void* out, long long ld_out,
                              int H, int h0, int Hn, int D, int V, int rank, int k_col, int v_col, int g_col, int a_col, float scale,
                              float inv_tau, float eps, int dt, void* stream_) {
  if (n_chunks <= 0 || n_reqs <= 0) return 0;
  if (H <= 0 || h0 < 0 || Hn <= 0 || h0 + Hn > H || Hn > 65535 || n_reqs > 65535 || D <= 0 || V <= 0 || D > 256 || V > 256 || D % 8 != 0 || V % 8 != 0 ||
      rank <= 0 || rank > GC_MAX_RANK || ld % 8 != 0 || k_col % 8 != 0 || v_col % 8 != 0 || g_col % 8 != 0 || ld_out % 2 != 0 ||
      (reinterpret_cast<uintptr_t>(proj) & 15) || (dt != 0 && dt != 1))
    return -1;
  GlaParams p = {};
  p.proj = proj; p.ld = ld; p.a2 = a2; p.a2_b = a2_b; p.norm_w = norm_w; p.state = state; p.chunks = chunks; p.n_chunks = n_chunks; p.reqs = reqs;
  p.inc = inc; p.dec = dec; p.out = out; p.ld_out = ld_out; p.H = H; p.h0 = h0; p.Hn = Hn; p.D = D; p.V = V; p.rank = rank; p.k_col = k_col;
  p.v_col = v_col; p.g_col = g_col; p.a_col = a_col; p.scale = scale; p.inv_tau = inv_tau; p.eps = eps;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  const int rp = (rank + 15) & ~15;
  const size_t sm_state = (size_t)(GC * gc_ld_state(D) + GC * rp + GC_THREADS) * 4 + (size_t)GC * gc_ld_v(V) * 2;
  const size_t sm_out = (size_t)(GC * gc_ld_out(D) + GC * GC_LD_A + GC_THREADS + 8 * GC) * 4 + (size_t)GC * (2 * gc_ld_qk(D) + gc_ld_v(V)) * 2;
  const dim3 grid(n_chunks, Hn), scan((D * V / 4 + 255) / 256, Hn, n_reqs);
  const int ntw = (V + 63) / 64;
#define LAUNCH(kern, gr, sm)                                                                                                     \
  {                                                                                                                             \
    static DeviceOnce cfg;                                                                                                      \
    if (cfg.need()) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);                        \
    launch_k(kern, gr, dim3(GC_THREADS), sm, stream, 0, p);                                                                     \
  }
  if (dt == 1) LAUNCH(gla_chunk_state_kernel<1>, grid, sm_state) else LAUNCH(gla_chunk_state_kernel<0>, grid, sm_state)
  launch_k(gla_chunk_scan_kernel, scan, dim3(256), 0, stream, 0, p);
#define OUT(NT) { if (dt == 1) LAUNCH((gla_chunk_out_kernel<1, NT>), grid, sm_out) else LAUNCH((gla_chunk_out_kernel<0, NT>), grid, sm_out) }
  if (ntw == 1) OUT(1) else if (ntw == 2) OUT(2) else if (ntw == 3) OUT(3) else OUT(4)
#undef OUT
#undef LAUNCH
  return (int)cudaGetLastError();
}
