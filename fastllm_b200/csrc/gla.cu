// Gated linear attention for sm_100a: per head a [D, V] fp32 state S whose key channels d forget at their own data-dependent rate.  A token
// with query q, key k, value v and decay logits z does
//     S[d, :] <- f[d] S[d, :] + k[d] v,   f[d] = sigmoid(z[d])^(1 / tau),   out = sum_d q[d] S[d, :],
// then comes the RMS norm of every head's output and * silu(gate).  z = W_a2 a + b comes from a low-rank row a.  q, k, v, gate and a_t are columns of one merged projection row.
//
//  * gla_recurrent_kernel: one CTA per (head, request) walks the request's tokens with the state in registers; a thread owns R rows of
//    one state column, so the state is read once and written once per step.  Any widths, fp32 included.
//  * the chunked form for prompts, 64 tokens per chunk, every chunk and head in parallel except for the scan:
//      gla_chunk_state   U_c = sum_t (k_t exp(b_C - b_t)) v_t^T         (the state's increment over the chunk; b: running log-decay)
//      gla_chunk_scan    S_c = exp(b_C) S_(c-1) + U_c                   (leaves S_(c-1) in place of U_c, the last one in the slot)
//      gla_chunk_out     o_t = S_(c-1)^T (q_t exp(b_t)) + sum_(s <= t) A_ts v_s,  A_ts = sum_d q_td k_sd exp(b_td - b_sd)
//    Queries are decayed from the start of their block of 16 tokens, keys to the end of theirs, so a product of two blocks needs one
//    more factor per channel: the decay between the blocks.  Inside a block that factor is the inverse of the block's decay; where it
//    would leave fp32's range (2^80) the block is taken pair by pair.  Every other exponent is a difference forwards in time and never
//    positive.  Products run on tf32 operands (q, k and the state carry ten fraction bits beyond which bf16 inputs have nothing left
//    but the decay factors) with fp32 accumulation; the state stays fp32.
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
  float* inc; float* dec; float* lg;       // [n_chunks, Hn, D, V], [n_chunks, Hn, D], [n_chunks, Hn, 64, D] running log2-decays
  int n_chunks, h0, Hn;
};

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
// the same to a few units in the last place without the library's logarithm: log(1 + e) = 2 artanh(e / (2 + e)), whose argument is at
// most 1/3, so seven terms of the series are enough
__device__ __forceinline__ float log_sigmoid_series(float z) {
  const float e = __expf(-fabsf(z)), x = __fdividef(e, 2.f + e), y = x * x;
  float t = fmaf(y, 1.f / 13.f, 1.f / 11.f);
  t = fmaf(y, t, 1.f / 9.f); t = fmaf(y, t, 1.f / 7.f); t = fmaf(y, t, 1.f / 5.f); t = fmaf(y, t, 1.f / 3.f); t = fmaf(y, t, 1.f);
  return fminf(z, 0.f) - 2.f * x * t;
}

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
      if (DT != 2 && (p.rank & 7) == 0) {
        for (int r = 0; r < p.rank; r += 8) {
          const uint4 wv = *reinterpret_cast<const uint4*>(w + r), av = *reinterpret_cast<const uint4*>(ar + r);
          const uint32_t wu[4] = {wv.x, wv.y, wv.z, wv.w}, au[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float2 a = unpack_16<DT == 1>(wu[i]), b = unpack_16<DT == 1>(au[i]);
            z = fmaf(a.x, b.x, z); z = fmaf(a.y, b.y, z);
          }
        }
      } else {
#pragma unroll 4
        for (int r = 0; r < p.rank; ++r) z = fmaf(GAct<DT>::ld(w[r]), GAct<DT>::ld(ar[r]), z);
      }
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
constexpr int GC_THREADS = 512;
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
constexpr int GC_LD_A = GC + 4;

// rows [row0, row0 + n) of `width` 16-bit columns into shared memory, zero rows behind them
__device__ __forceinline__ void gc_load(const uint16_t* src, long long ld, int n, int width, uint16_t* dst, int ld_dst) {
  const int vecs = width >> 3;
  for (int i = threadIdx.x; i < GC * vecs; i += blockDim.x) {
    const int t = i / vecs, c = (i - t * vecs) << 3;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (t < n) v = *reinterpret_cast<const uint4*>(src + (size_t)t * ld + c);
    *reinterpret_cast<uint4*>(dst + (size_t)t * ld_dst + c) = v;
  }
}

// DS > 0: D = V = DS known at compile time
template <int DT, int DS>
__global__ void __launch_bounds__(GC_THREADS, 2) gla_chunk_state_kernel(const GlaParams p) {
  extern __shared__ float sm[];
  const int D = DS > 0 ? DS : p.D, V = DS > 0 ? DS : p.V, ldb = gc_ld_state(D), ldv = gc_ld_v(V), rp = (p.rank + 7) & ~7, lda = rp + 4;
  float* kt = sm;                                                     // [GC][ldb] log-decays, then decayed keys
  float* a1 = kt + GC * ldb;                                          // [GC][lda]
  float* tot = a1 + GC * lda;                                         // [GC_THREADS]
  uint16_t* vs = reinterpret_cast<uint16_t*>(tot + GC_THREADS);       // [GC][ldv]
  const int c = blockIdx.x, hl = blockIdx.y, h = p.h0 + hl;
  const int r0 = p.chunks[2 * c], n = p.chunks[2 * c + 1];
  const uint16_t* row0 = reinterpret_cast<const uint16_t*>(p.proj) + (size_t)r0 * p.ld;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  gc_load(row0 + p.v_col + h * V, p.ld, n, V, vs, ldv);
  for (int i = threadIdx.x; i < GC * rp; i += GC_THREADS) {
    const int t = i / rp, x = i - t * rp;
    a1[t * lda + x] = (t < n && x < p.rank) ? GAct<DT>::ld(row0[(size_t)t * p.ld + p.a_col + x]) : 0.f;
  }
  __syncthreads();
  // log2-decays of single tokens: z = a W_a2^T + b on the tensor core (16-bit factors are exact in tf32)
  const uint16_t* a2 = reinterpret_cast<const uint16_t*>(p.a2) + (size_t)h * D * p.rank;
  const uint16_t* ab = reinterpret_cast<const uint16_t*>(p.a2_b) + (size_t)h * D;
  for (int nt = warp; nt < (D >> 3); nt += GC_THREADS / 32) {
    float acc[4][4] = {};
    for (int k0 = 0; k0 < rp; k0 += 8) {
      const uint16_t* w = a2 + (size_t)(nt * 8 + g) * p.rank + k0 + q;
      const float b0 = k0 + q < p.rank ? GAct<DT>::ld(w[0]) : 0.f, b1 = k0 + q + 4 < p.rank ? GAct<DT>::ld(w[4]) : 0.f;
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const float* ap = a1 + (16 * m + g) * lda + k0 + q;
        const float a[4] = {ap[0], ap[8 * lda], ap[4], ap[8 * lda + 4]};
        mma_tf32(acc[m], a, b0, b1);
      }
    }
    const int d = nt * 8 + 2 * q;
    const float z0 = GAct<DT>::ld(ab[d]), z1 = GAct<DT>::ld(ab[d + 1]), f = p.inv_tau * 1.4426950408889634f;
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
      for (int hf = 0; hf < 2; ++hf) {
        const int t = 16 * m + 8 * hf + g;                            // (rows beyond n decay by nothing)
        const float x = log_sigmoid_series(acc[m][2 * hf] + z0) * f, y = log_sigmoid_series(acc[m][2 * hf + 1] + z1) * f;
        *reinterpret_cast<float2*>(kt + t * ldb + d) = t < n ? make_float2(x, y) : make_float2(0.f, 0.f);
      }
  }
  __syncthreads();
  // running sums per channel, in parts of the chunk; then the decayed keys in their place
  const int parts = D <= 64 ? 8 : D <= 128 ? 4 : 2, tp = GC / parts, wd = GC_THREADS / parts;
  const int part = threadIdx.x / wd, d = threadIdx.x - part * wd;
  float run = 0.f;
  if (d < D) {
    float* col = kt + part * tp * ldb + d;
#pragma unroll 8
    for (int t = 0; t < tp; ++t) { run += col[t * ldb]; col[t * ldb] = run; }
  }
  tot[threadIdx.x] = run;
  __syncthreads();
  const uint16_t* kp = row0 + p.k_col + h * D;
  const size_t unit = (size_t)c * p.Hn + hl;
  if (d < D) {
    float off = 0.f, last = 0.f;
    for (int i = 0; i < parts; ++i) { const float x = tot[i * wd + d]; last += x; if (i < part) off += x; }
    if (part == 0) p.dec[unit * D + d] = ex2(last);
    float* lg = p.lg + unit * GC * D + d;
#pragma unroll 4
    for (int t = part * tp; t < (part + 1) * tp; ++t) {
      const float b = kt[t * ldb + d] + off;
      const float k = t < n ? GAct<DT>::ld(kp[(size_t)t * p.ld + d]) : 0.f;
      lg[(size_t)t * D] = b;
      kt[t * ldb + d] = to_tf32(k * ex2(last - b));
    }
  }
  __syncthreads();
  // U[d][v] = sum_t K~[t][d] V[t][v]: a warp takes 16 rows x 64 columns
  const int mbs = (D + 15) >> 4, nts = V >> 3, ngs = (nts + 7) >> 3;
  float* U = p.inc + unit * D * V;
  for (int u = warp; u < mbs * ngs; u += GC_THREADS / 32) {
    const int mb = u % mbs, nt0 = (u / mbs) * 8, cnt = min(8, nts - nt0);
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i) { acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f; }
#pragma unroll 2
    for (int k0 = 0; k0 < GC; k0 += 8) {
      const float* ap = kt + (k0 + q) * ldb + mb * 16 + g;            // (columns beyond D: the row's padding, never stored)
      const float a[4] = {ap[0], ap[8], ap[4 * ldb], ap[4 * ldb + 8]};
      const uint16_t* bp = vs + (k0 + q) * ldv + nt0 * 8 + g;
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (i < cnt) mma_tf32(acc[i], a, GAct<DT>::ld(bp[i * 8]), GAct<DT>::ld(bp[4 * ldv + i * 8]));
    }
    const int d0 = mb * 16 + g;
    float* up = U + (size_t)d0 * V + nt0 * 8 + 2 * q;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (i >= cnt) break;
      if (d0 < D) *reinterpret_cast<float2*>(up + i * 8) = make_float2(acc[i][0], acc[i][1]);
      if (d0 + 8 < D) *reinterpret_cast<float2*>(up + 8 * V + i * 8) = make_float2(acc[i][2], acc[i][3]);
    }
  }
}

// one thread per two state elements of a (request, head); reads run ahead of the dependent chain
__global__ void __launch_bounds__(128) gla_chunk_scan_kernel(const GlaParams p) {
  const int D = p.D, V = p.V, hl = blockIdx.y;
  const int e = (blockIdx.x * 128 + threadIdx.x) * 2;
  if (e >= D * V) return;
  const int c0 = p.reqs[3 * blockIdx.z], n = p.reqs[3 * blockIdx.z + 1], slot = p.reqs[3 * blockIdx.z + 2];
  const int d = e / V;
  float2* st = reinterpret_cast<float2*>(p.state + ((size_t)slot * p.H + p.h0 + hl) * D * V + e);
  float2 s = *st;
  const size_t su = (size_t)p.Hn * D * V, sd = (size_t)p.Hn * D;
  float* U = p.inc + ((size_t)c0 * p.Hn + hl) * D * V + e;
  const float* dc = p.dec + ((size_t)c0 * p.Hn + hl) * D + d;
  constexpr int A = 8;
  float2 u[2][A];
  float f[2][A];
  auto fetch = [&](int k, int c) {
#pragma unroll
    for (int i = 0; i < A; ++i)
      if (c + i < n) { u[k][i] = *reinterpret_cast<const float2*>(U + (size_t)(c + i) * su); f[k][i] = dc[(size_t)(c + i) * sd]; }
  };
  auto step = [&](int k, int c) {
#pragma unroll
    for (int i = 0; i < A; ++i) {
      if (c + i >= n) break;
      *reinterpret_cast<float2*>(U + (size_t)(c + i) * su) = s;
      s.x = fmaf(s.x, f[k][i], u[k][i].x); s.y = fmaf(s.y, f[k][i], u[k][i].y);
    }
  };
  fetch(0, 0);
  for (int c = 0; c < n; c += 2 * A) {
    fetch(1, c + A);
    step(0, c);
    fetch(0, c + 2 * A);
    step(1, c + A);
  }
  *st = s;
}

// NTW: 8-column output tiles per warp, ceil(V / 64); the first eight warps take rows 0..31 of the output, the others 32..63
template <int DT, int NTW, int DS>
__global__ void __launch_bounds__(GC_THREADS, NTW <= 2 ? 2 : 1) gla_chunk_out_kernel(const GlaParams p) {
  extern __shared__ float sm[];
  const int D = DS > 0 ? DS : p.D, V = DS > 0 ? DS : p.V, ldb = gc_ld_out(D), ldv = gc_ld_v(V);
  float* qh = sm;                                                     // [GC][ldb] log-decays, then decayed queries
  float* kh = qh + GC * ldb;                                          // [GC][ldb] decayed keys
  float* At = kh + GC * ldb;                                          // [GC][GC_LD_A]
  float* edge = At + GC * GC_LD_A;                                    // [5][ldb] log-decay at the start of block 0..3 and at the end
  float* red = edge + 5 * ldb;                                        // [8][GC] partial squares, [GC] norms
  uint16_t* vs = reinterpret_cast<uint16_t*>(red + 9 * GC);           // [GC][ldv]
  const int c = blockIdx.x, hl = blockIdx.y, h = p.h0 + hl;
  const int r0 = p.chunks[2 * c], n = p.chunks[2 * c + 1];
  const uint16_t* row0 = reinterpret_cast<const uint16_t*>(p.proj) + (size_t)r0 * p.ld;
  const uint16_t* qrow = row0 + h * D;
  const uint16_t* krow = row0 + p.k_col + h * D;
  gc_load(row0 + p.v_col + h * V, p.ld, n, V, vs, ldv);
  const float* lg = p.lg + ((size_t)c * p.Hn + hl) * GC * D;
  const int dv = D >> 2;
  for (int i = threadIdx.x; i < GC * dv; i += GC_THREADS) {
    const int t = i / dv, d = (i - t * dv) << 2;
    *reinterpret_cast<float4*>(qh + t * ldb + d) = *reinterpret_cast<const float4*>(lg + (size_t)t * D + d);
  }
  for (int i = threadIdx.x; i < GC * GC_LD_A; i += GC_THREADS) At[i] = 0.f;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3;
  bool wide = false;                                                  // some channel of some block decays beyond the factored form
  for (int d = threadIdx.x; d < D; d += GC_THREADS) {
    float e = 0.f;
    edge[d] = 0.f;
#pragma unroll
    for (int i = 1; i < 5; ++i) {
      const float nx = qh[(16 * i - 1) * ldb + d];
      wide = wide || e - nx > 80.f;
      edge[i * ldb + d] = e = nx;
    }
  }
  const bool pairs = __syncthreads_or(wide);
  if (pairs) {
    // A inside a block pair by pair, a row of every block per warp
    for (int blk = 0; blk < 4; ++blk) {
      const int t = 16 * blk + ((blk & 1) ? 15 - warp : warp);
      if (t >= n) continue;
      for (int s = 16 * blk; s <= t; ++s) {
        float x = 0.f;
        for (int d = lane; d < D; d += 32)
          x = fmaf(GAct<DT>::ld(qrow[(size_t)t * p.ld + d]) * GAct<DT>::ld(krow[(size_t)s * p.ld + d]), ex2(qh[t * ldb + d] - qh[s * ldb + d]), x);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
        if (lane == 0) At[t * GC_LD_A + s] = to_tf32(x * p.scale);
      }
    }
    __syncthreads();
  }
  // queries decayed from the start of their block, keys to the end of theirs
  for (int i = threadIdx.x; i < GC * dv; i += GC_THREADS) {
    const int t = i / dv, d = (i - t * dv) << 2;
    const float4 b = *reinterpret_cast<const float4*>(qh + t * ldb + d);
    const float4 e0 = *reinterpret_cast<const float4*>(edge + (t >> 4) * ldb + d), e1 = *reinterpret_cast<const float4*>(edge + ((t >> 4) + 1) * ldb + d);
    float4 qv = make_float4(0.f, 0.f, 0.f, 0.f), kv = qv;
    if (t < n) {
      const uint2 qu = *reinterpret_cast<const uint2*>(qrow + (size_t)t * p.ld + d), ku = *reinterpret_cast<const uint2*>(krow + (size_t)t * p.ld + d);
      const float2 q0 = unpack_16<DT == 1>(qu.x), q1 = unpack_16<DT == 1>(qu.y), k0 = unpack_16<DT == 1>(ku.x), k1 = unpack_16<DT == 1>(ku.y);
      qv = make_float4(to_tf32(q0.x * p.scale * ex2(b.x - e0.x)), to_tf32(q0.y * p.scale * ex2(b.y - e0.y)), to_tf32(q1.x * p.scale * ex2(b.z - e0.z)),
                       to_tf32(q1.y * p.scale * ex2(b.w - e0.w)));
      kv = make_float4(to_tf32(k0.x * ex2(e1.x - b.x)), to_tf32(k0.y * ex2(e1.y - b.y)), to_tf32(k1.x * ex2(e1.z - b.z)), to_tf32(k1.y * ex2(e1.w - b.w)));
    }
    *reinterpret_cast<float4*>(qh + t * ldb + d) = qv;
    *reinterpret_cast<float4*>(kh + t * ldb + d) = kv;
  }
  __syncthreads();
  // A block by block: 6 pairs of different blocks, then the 4 diagonal ones
  for (int u = warp; u < (pairs ? 6 : 10); u += GC_THREADS / 32) {
    const int i = u >= 6 ? u - 6 : u < 1 ? 1 : u < 3 ? 2 : 3, j = u >= 6 ? i : u - (i * (i - 1)) / 2;
    const float *ei = edge + i * ldb + q, *ej = edge + (j + 1) * ldb + q;       // the factor between them: exp2(ei - ej)
    const float* qp = qh + (16 * i + g) * ldb + q;
    const float* kp = kh + (16 * j + g) * ldb + q;
    float acc[2][4] = {};
#pragma unroll 4
    for (int k0 = 0; k0 < D; k0 += 8) {
      float a[4] = {qp[k0], qp[8 * ldb + k0], qp[k0 + 4], qp[8 * ldb + k0 + 4]};
      if (j + 1 != i) {
        const float f0 = ex2(ei[k0] - ej[k0]), f1 = ex2(ei[k0 + 4] - ej[k0 + 4]);
        a[0] = to_tf32(a[0] * f0); a[1] = to_tf32(a[1] * f0); a[2] = to_tf32(a[2] * f1); a[3] = to_tf32(a[3] * f1);
      }
      mma_tf32(acc[0], a, kp[k0], kp[k0 + 4]);
      mma_tf32(acc[1], a, kp[8 * ldb + k0], kp[8 * ldb + k0 + 4]);
    }
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = g + (e >> 1) * 8, s = m * 8 + 2 * q + (e & 1);
        At[(16 * i + t) * GC_LD_A + 16 * j + s] = (i != j || s <= t) ? to_tf32(acc[m][e]) : 0.f;
      }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < (GC - 16) * dv; i += GC_THREADS) {          // queries decayed from the start of the chunk (block 0 is)
    const int t = 16 + i / dv, d = (i - (t - 16) * dv) << 2;
    const float4 e0 = *reinterpret_cast<const float4*>(edge + (t >> 4) * ldb + d);
    float4 b = *reinterpret_cast<float4*>(qh + t * ldb + d);
    b.x = to_tf32(b.x * ex2(e0.x)); b.y = to_tf32(b.y * ex2(e0.y)); b.z = to_tf32(b.z * ex2(e0.z)); b.w = to_tf32(b.w * ex2(e0.w));
    *reinterpret_cast<float4*>(qh + t * ldb + d) = b;
  }
  __syncthreads();
  // O = Q~ S + A V
  const float* S = p.inc + ((size_t)c * p.Hn + hl) * D * V;
  const int half = warp >> 3, cw = warp & 7, m0 = 32 * half;
  float acc[2][NTW][4];
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int i = 0; i < NTW; ++i) { acc[m][i][0] = acc[m][i][1] = acc[m][i][2] = acc[m][i][3] = 0.f; }
  const int v0 = cw * NTW * 8;
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
    for (int m = 0; m < 2; ++m) {
      const float* ap = qh + (m0 + 16 * m + g) * ldb + k0 + q;
      const float a[4] = {ap[0], ap[8 * ldb], ap[4], ap[8 * ldb + 4]};
#pragma unroll
      for (int i = 0; i < NTW; ++i) mma_tf32(acc[m][i], a, to_tf32(b0[i]), to_tf32(b1[i]));
    }
  }
#pragma unroll 2
  for (int k0 = 0; k0 < m0 + 32; k0 += 8) {                           // (beyond: above the diagonal)
    float b0[NTW], b1[NTW];
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
      const int v = v0 + i * 8 + g;
      b0[i] = v < V ? GAct<DT>::ld(vs[(k0 + q) * ldv + v]) : 0.f;
      b1[i] = v < V ? GAct<DT>::ld(vs[(k0 + q + 4) * ldv + v]) : 0.f;
    }
#pragma unroll
    for (int m = 0; m < 2; ++m) {
      const float* ap = At + (m0 + 16 * m + g) * GC_LD_A + k0 + q;
      const float a[4] = {ap[0], ap[8 * GC_LD_A], ap[4], ap[8 * GC_LD_A + 4]};
#pragma unroll
      for (int i = 0; i < NTW; ++i) mma_tf32(acc[m][i], a, b0[i], b1[i]);
    }
  }
  // norm over the head's V columns, weight, gate
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
      s0 += acc[m][i][0] * acc[m][i][0] + acc[m][i][1] * acc[m][i][1];
      s1 += acc[m][i][2] * acc[m][i][2] + acc[m][i][3] * acc[m][i][3];
    }
    s0 += __shfl_xor_sync(0xffffffffu, s0, 1); s0 += __shfl_xor_sync(0xffffffffu, s0, 2);
    s1 += __shfl_xor_sync(0xffffffffu, s1, 1); s1 += __shfl_xor_sync(0xffffffffu, s1, 2);
    if (q == 0) { red[cw * GC + m0 + 16 * m + g] = s0; red[cw * GC + m0 + 16 * m + 8 + g] = s1; }
  }
  __syncthreads();
  if (threadIdx.x < GC) {
    float ss = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) ss += red[w * GC + threadIdx.x];
    red[8 * GC + threadIdx.x] = 1.0f / sqrtf(ss / (float)V + p.eps);
  }
  __syncthreads();
  const uint16_t* nw = reinterpret_cast<const uint16_t*>(p.norm_w);
#pragma unroll
  for (int m = 0; m < 2; ++m) {
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int t = m0 + 16 * m + 8 * hf + g;
      if (t >= n) continue;
      const float inv = red[8 * GC + t];
      const uint16_t* gp = row0 + (size_t)t * p.ld + p.g_col + h * V;
      uint16_t* op = reinterpret_cast<uint16_t*>(p.out) + (size_t)(r0 + t) * p.ld_out + (size_t)h * V;
#pragma unroll
      for (int i = 0; i < NTW; ++i) {
        const int v = v0 + i * 8 + 2 * q;
        if (v >= V) continue;
        const float2 gv = unpack_16<DT == 1>(*reinterpret_cast<const uint32_t*>(gp + v));
        const float2 wv = unpack_16<DT == 1>(*reinterpret_cast<const uint32_t*>(nw + v));
        const float y0 = acc[m][i][2 * hf] * inv * wv.x * __fdividef(gv.x, 1.0f + __expf(-gv.x));
        const float y1 = acc[m][i][2 * hf + 1] * inv * wv.y * __fdividef(gv.y, 1.0f + __expf(-gv.y));
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
  if (dt != 2 && rank % 8 == 0 && ((ld % 8) || (a_col % 8) || (reinterpret_cast<uintptr_t>(proj) & 15) || (reinterpret_cast<uintptr_t>(a2) & 15))) return -1;
  GlaParams p = {};
  p.proj = proj; p.ld = ld; p.a2 = a2; p.a2_b = a2_b; p.norm_w = norm_w; p.state = state; p.slots = slots; p.cu = cu; p.out = out; p.ld_out = ld_out;
  p.H = H; p.D = D; p.V = V; p.rank = rank; p.k_col = k_col; p.v_col = v_col; p.g_col = g_col; p.a_col = a_col;
  p.scale = scale; p.inv_tau = inv_tau; p.eps = eps;
  const int cgs = (V + 31) / 32;
  int R = 0, rgs = 1;
  for (int warps = 8; warps <= 16 && R == 0; warps *= 2)       // 256 threads where the state fits their registers, else 512
    for (int r = 16; r <= 64; r *= 2) {
      const int g = (D + r - 1) / r;
      if (cgs * g <= warps) { R = r; rgs = g; break; }
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
// and lg [n_chunks * Hn * 64 * D] floats.  16-bit projections, D and V multiples of 8 up to 256, rank up to 64.
extern "C" int fb_gla_chunked(const void* proj, long long ld, const void* a2, const void* a2_b, const void* norm_w, float* state,
                              const int* chunks, int n_chunks, const int* reqs, int n_reqs, float* inc, float* dec, float* lg, void* out, long long ld_out,
                              int H, int h0, int Hn, int D, int V, int rank, int k_col, int v_col, int g_col, int a_col, float scale,
                              float inv_tau, float eps, int dt, void* stream_) {
  if (n_chunks <= 0 || n_reqs <= 0) return 0;
  if (H <= 0 || h0 < 0 || Hn <= 0 || h0 + Hn > H || Hn > 65535 || n_reqs > 65535 || D <= 0 || V <= 0 || D > 256 || V > 256 || D % 8 != 0 || V % 8 != 0 ||
      rank <= 0 || rank > GC_MAX_RANK || ld % 8 != 0 || k_col % 8 != 0 || v_col % 8 != 0 || g_col % 8 != 0 || ld_out % 2 != 0 ||
      (reinterpret_cast<uintptr_t>(proj) & 15) || (dt != 0 && dt != 1))
    return -1;
  GlaParams p = {};
  p.proj = proj; p.ld = ld; p.a2 = a2; p.a2_b = a2_b; p.norm_w = norm_w; p.state = state; p.chunks = chunks; p.n_chunks = n_chunks; p.reqs = reqs;
  p.inc = inc; p.dec = dec; p.lg = lg; p.out = out; p.ld_out = ld_out; p.H = H; p.h0 = h0; p.Hn = Hn; p.D = D; p.V = V; p.rank = rank; p.k_col = k_col;
  p.v_col = v_col; p.g_col = g_col; p.a_col = a_col; p.scale = scale; p.inv_tau = inv_tau; p.eps = eps;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  const size_t sm_state = (size_t)(GC * gc_ld_state(D) + GC * (((rank + 7) & ~7) + 4) + GC_THREADS) * 4 + (size_t)GC * gc_ld_v(V) * 2;
  const size_t sm_out = (size_t)((2 * GC + 5) * gc_ld_out(D) + GC * GC_LD_A + 9 * GC) * 4 + (size_t)GC * gc_ld_v(V) * 2;
  const dim3 grid(n_chunks, Hn), scan((D * V / 2 + 127) / 128, Hn, n_reqs);
  const int ntw = (V + 63) / 64;
#define LAUNCH(kern, gr, sm)                                                                                                     \
  {                                                                                                                             \
    static DeviceOnce cfg;                                                                                                      \
    if (cfg.need()) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);                        \
    launch_k(kern, gr, dim3(GC_THREADS), sm, stream, 0, p);                                                                     \
  }
  const bool std128 = D == 128 && V == 128;
#define STATE(DS) { if (dt == 1) LAUNCH((gla_chunk_state_kernel<1, DS>), grid, sm_state) else LAUNCH((gla_chunk_state_kernel<0, DS>), grid, sm_state) }
  if (std128) STATE(128) else STATE(0)
#undef STATE
  launch_k(gla_chunk_scan_kernel, scan, dim3(128), 0, stream, 0, p);
#define OUT(NT, DS) { if (dt == 1) LAUNCH((gla_chunk_out_kernel<1, NT, DS>), grid, sm_out) else LAUNCH((gla_chunk_out_kernel<0, NT, DS>), grid, sm_out) }
  if (std128) OUT(2, 128) else if (ntw == 1) OUT(1, 0) else if (ntw == 2) OUT(2, 0) else if (ntw == 3) OUT(3, 0) else OUT(4, 0)
#undef OUT
#undef LAUNCH
  return (int)cudaGetLastError();
}
