// 32-bit and any-size forms of a model's matrix products, of latent attention and of grouped-query attention (CUDA cores, fp32 FMAs).
//
// They serve models run in float32, where the tensor core has no full-precision mode, and 16-bit shapes outside the tensor-core
// kernels' tiling.  Compiled without fast-math.
#include "ptx.cuh"
#include "launch.h"

FB_DEFINE_ERROR_API(full32)

namespace fb {

template <int DT> struct F32In;
template <> struct F32In<0> { typedef uint16_t T; static __device__ __forceinline__ float ld(uint16_t v) { return __half2float(__ushort_as_half(v)); }
                              static __device__ __forceinline__ uint16_t st(float v) { return __half_as_ushort(__float2half_rn(v)); } };
template <> struct F32In<1> { typedef uint16_t T; static __device__ __forceinline__ float ld(uint16_t v) { return __bfloat162float(__ushort_as_bfloat16(v)); }
                              static __device__ __forceinline__ uint16_t st(float v) { return __bfloat16_as_ushort(__float2bfloat16_rn(v)); } };
template <> struct F32In<2> { typedef float T; static __device__ __forceinline__ float ld(float v) { return v; } static __device__ __forceinline__ float st(float v) { return v; } };

// out[m, n] = act(sum_k X[m, k] W[n, k]) (* sigmoid(gate[m, n])), or residual[m, n] + alpha * (...) in fp32.
// blockIdx.z selects a batch (its own weight rows, column slices of X and out) or, with `counts`, an expert and its segment of rows.
struct Full32Params {
  const void* X; const void* W; void* out;
  const float* residual; const void* gate; const void* bias;
  int M, N, K;
  long long ldx, ldw, ld_out, ld_res, ld_gate;
  long long batch_w_rows, batch_x_cols, batch_out_cols;
  const int* counts; const int* offsets;
  float alpha;
  int act, out_f32;                        // act: 0 none, 1 relu^2, 2 gelu (erf), 3 gelu (tanh form)
  // factors of the activated product: sigmoid of one fp32 logit per row; row mul_rows[m] of a table
  const float* row_gate; long long ld_row_gate;
  const void* mul; const int* mul_rows; long long ld_mul; int mul_count;
};

__device__ __forceinline__ float act32(float v, int act) {
  if (act == 1) { v = fmaxf(v, 0.f); return v * v; }
  if (act == 2) return 0.5f * v * (1.0f + erff(v * 0.70710678118654752f));
  if (act == 3) return 0.5f * v * (1.0f + tanhf(0.79788456080286536f * (v + 0.044715f * v * v * v)));
  return v;
}

template <int DT>
__global__ void __launch_bounds__(256) gemm_full32_kernel(const Full32Params p) {
  typedef typename F32In<DT>::T T;
  constexpr int BM = 64, BN = 64, BK = 16;
  __shared__ float xs[BK][BM + 4], ws[BK][BN + 4];
  const int z = blockIdx.z;
  int M = p.M;
  long long row0 = 0;
  if (p.counts != nullptr) { M = p.counts[z]; row0 = p.offsets[z]; }
  const int n0 = blockIdx.x * BN;
  const T* X = reinterpret_cast<const T*>(p.X) + z * p.batch_x_cols;
  const T* W = reinterpret_cast<const T*>(p.W) + z * p.batch_w_rows * p.ldw;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  for (int m0 = blockIdx.y * BM; m0 < M; m0 += gridDim.y * BM) {
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < p.K; k0 += BK) {
      for (int i = threadIdx.x; i < BM * BK; i += 256) {
        const int r = i / BK, k = i - r * BK;
        const bool in_k = k0 + k < p.K;
        xs[k][r] = (in_k && m0 + r < M) ? F32In<DT>::ld(X[(row0 + m0 + r) * p.ldx + k0 + k]) : 0.f;
        ws[k][r] = (in_k && n0 + r < p.N) ? F32In<DT>::ld(W[(long long)(n0 + r) * p.ldw + k0 + k]) : 0.f;
      }
      __syncthreads();
#pragma unroll
      for (int k = 0; k < BK; ++k) {
        float a[4], b[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) { a[i] = xs[k][ty * 4 + i]; b[i] = ws[k][tx * 4 + i]; }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
      }
      __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int m = m0 + ty * 4 + i;
      if (m >= M) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int n = n0 + tx * 4 + j;
        if (n >= p.N) continue;
        float v = acc[i][j];
        const long long c = z * p.batch_out_cols + n;
        if (p.bias != nullptr) v += F32In<DT>::ld(reinterpret_cast<const T*>(p.bias)[n]);
        v = act32(v, p.act);
        if (p.row_gate != nullptr) v *= 1.0f / (1.0f + expf(-p.row_gate[(row0 + m) * p.ld_row_gate]));
        if (p.mul != nullptr) v *= F32In<DT>::ld(reinterpret_cast<const T*>(p.mul)[min(max(p.mul_rows[row0 + m], 0), p.mul_count - 1) * p.ld_mul + n]);
        if (p.gate != nullptr) v *= 1.0f / (1.0f + expf(-F32In<DT>::ld(reinterpret_cast<const T*>(p.gate)[(row0 + m) * p.ld_gate + c])));
        if (p.residual != nullptr) v = p.residual[(row0 + m) * p.ld_res + c] + p.alpha * v;
        if (p.out_f32) reinterpret_cast<float*>(p.out)[(row0 + m) * p.ld_out + c] = v;
        else reinterpret_cast<T*>(p.out)[(row0 + m) * p.ld_out + c] = F32In<DT>::st(v);
      }
    }
  }
}

// Latent attention of one (row, head) per CTA over the paged latent cache, any latent width:
//   score[j] = scale * q[row, head] . c[j],  out = sum_j softmax(score)[j] c[j][:RV],  first <= j <= position
// where R >= RV: what follows a row's values takes part in the scores alone (a rotated key part).  head_gate: one fp32 logit per head.
// 128 threads: a warp scores one key at a time (lanes over the latent), then every thread accumulates its latent columns.
constexpr int L32_KEYS = 64;
template <int DT>
__global__ void __launch_bounds__(128) latent_attn32_kernel(const typename F32In<DT>::T* __restrict__ q, const typename F32In<DT>::T* __restrict__ pool,
                                                            typename F32In<DT>::T* __restrict__ out, const int* __restrict__ page_table,
                                                            const int* __restrict__ kv_lens, int max_pages, int page_len, int H, int R,
                                                            int RV, int ld, int window, float scale, const float* __restrict__ head_gate) {
  extern __shared__ float sm[];
  float* qs = sm;                       // [R]
  float* os = sm + R;                   // [RV] running output
  __shared__ float sc[L32_KEYS];
  __shared__ int rows[L32_KEYS];
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n = kv_lens[t];
  const int first = (window > 0 && n > window) ? n - window : 0;
  const typename F32In<DT>::T* qp = q + ((size_t)t * H + h) * ld;
  for (int i = tid; i < R; i += 128) qs[i] = F32In<DT>::ld(qp[i]);
  for (int i = tid; i < RV; i += 128) os[i] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;
  for (int j0 = first; j0 < n; j0 += L32_KEYS) {
    const int cnt = n - j0 < L32_KEYS ? n - j0 : L32_KEYS;
    __syncthreads();
    if (tid < cnt) {
      const int j = j0 + tid, pg = j / page_len;
      rows[tid] = pg < max_pages ? page_table[(size_t)t * max_pages + pg] * page_len + (j - pg * page_len) : 0;
    }
    __syncthreads();
    for (int j = warp; j < cnt; j += 4) {
      const typename F32In<DT>::T* c = pool + (size_t)rows[j] * ld;
      float s = 0.f;
      for (int i = lane; i < R; i += 32) s = fmaf(qs[i], F32In<DT>::ld(c[i]), s);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (lane == 0) sc[j] = s * scale;
    }
    __syncthreads();
    float mx = m_run;
    for (int j = 0; j < cnt; ++j) mx = fmaxf(mx, sc[j]);
    const float fac = m_run == -INFINITY ? 0.f : expf(m_run - mx);
    __syncthreads();
    if (tid < cnt) sc[tid] = expf(sc[tid] - mx);
    __syncthreads();
    float l = 0.f;
    for (int j = 0; j < cnt; ++j) l += sc[j];
    l_run = l_run * fac + l;
    m_run = mx;
    for (int i = tid; i < RV; i += 128) {
      float a = os[i] * fac;
      for (int j = 0; j < cnt; ++j) a = fmaf(sc[j], F32In<DT>::ld(pool[(size_t)rows[j] * ld + i]), a);
      os[i] = a;
    }
  }
  float inv = l_run > 0.f ? 1.0f / l_run : 0.f;
  if (head_gate != nullptr) inv *= 1.0f / (1.0f + expf(-head_gate[(size_t)t * H + h]));
  typename F32In<DT>::T* op = out + ((size_t)t * H + h) * RV;
  for (int i = tid; i < RV; i += 128) op[i] = F32In<DT>::st(os[i] * inv);
}

// Grouped-query attention of one (row, query head) per CTA over paged keys and values, any widths, fp32 arithmetic:
//   out = (sum_j softmax(score_j) v_j) * sigmoid(gate),  score_j = scale q . k_j, soft-capped where the layer does
// Row t sees the keys of its own page-table row; its position is kv_lens[t] - 1.  The first key: chunk: position - position % chunk;
// window: position - window + 1, beside the first `keep` of the sequence; neither: 0.  sinks: one more term exp(sink) per head in the
// denominator.  The gate is elementwise (`gate`, 16-bit or fp32) or one fp32 logit per head (`head_gate`).  score_bias: the weights are
// sigmoid(score + score_bias[h]) and not normalised.  rot_v: the leading dimensions of the output, in pairs (2m, 2m + 1), are turned
// back by the row's position (tables [tab_rows, rot_v / 2]) before any gate.
struct Grouped32Params {
  const void* q; const void* k_pool; const void* v_pool; void* out; const void* gate;
  long long ld_q, ld_out, ld_gate;
  const int* page_table; const int* kv_lens;
  int H, G, D, Dp, Vp, max_pages, num_pages, page_len, window, chunk, keep;
  float scale, softcap;
  const float* sinks;
  const float* head_gate; long long ld_head_gate;
  const float* score_bias;
  const float* cos_v; const float* sin_v;
  int rot_v, tab_rows;
};

template <int DT>
__global__ void __launch_bounds__(128) grouped_attn32_kernel(const Grouped32Params p) {
  typedef typename F32In<DT>::T T;
  extern __shared__ float sm[];
  float* qs = sm;                       // [Dp]
  float* os = sm + p.Dp;                // [Vp] running output
  __shared__ float sc[L32_KEYS];
  __shared__ int rows[L32_KEYS];
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = h / (p.H / p.G);
  const int n = p.kv_lens[t], pos = n - 1;
  int first = 0;
  if (p.chunk > 0) first = n > 0 ? pos - pos % p.chunk : 0;
  else if (p.window > 0 && n > p.window) first = n - p.window;
  const T* qp = reinterpret_cast<const T*>(p.q) + (size_t)t * p.ld_q + (size_t)h * p.Dp;
  const T* kp = reinterpret_cast<const T*>(p.k_pool);
  const T* vp = reinterpret_cast<const T*>(p.v_pool);
  for (int i = tid; i < p.Dp; i += 128) qs[i] = F32In<DT>::ld(qp[i]);
  for (int i = tid; i < p.Vp; i += 128) os[i] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;
  const int kept = p.keep < first ? p.keep : first, keys = kept + n - first;       // keys 0 .. kept - 1 and first .. n - 1
  for (int j0 = 0; j0 < keys; j0 += L32_KEYS) {
    const int cnt = keys - j0 < L32_KEYS ? keys - j0 : L32_KEYS;
    __syncthreads();
    if (tid < cnt) {
      const int i = j0 + tid, j = i < kept ? i : first + i - kept, pg = j / p.page_len;
      int page = pg < p.max_pages ? p.page_table[(size_t)t * p.max_pages + pg] : 0;
      if ((unsigned)page >= (unsigned)p.num_pages) page = 0;
      rows[tid] = page * p.page_len + (j - pg * p.page_len);
    }
    __syncthreads();
    for (int j = warp; j < cnt; j += 4) {
      const T* c = kp + ((size_t)rows[j] * p.G + g) * p.Dp;
      float s = 0.f;
      for (int i = lane; i < p.D; i += 32) s = fmaf(qs[i], F32In<DT>::ld(c[i]), s);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      s *= p.scale;
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      if (lane == 0) sc[j] = p.score_bias != nullptr ? 1.0f / (1.0f + expf(-(s + p.score_bias[h]))) : s;
    }
    __syncthreads();
    float fac = 1.f;
    if (p.score_bias == nullptr) {
      float mx = m_run;
      for (int j = 0; j < cnt; ++j) mx = fmaxf(mx, sc[j]);
      fac = m_run == -INFINITY ? 0.f : expf(m_run - mx);
      __syncthreads();
      if (tid < cnt) sc[tid] = expf(sc[tid] - mx);
      __syncthreads();
      float l = 0.f;
      for (int j = 0; j < cnt; ++j) l += sc[j];
      l_run = l_run * fac + l;
      m_run = mx;
    }
    for (int i = tid; i < p.Vp; i += 128) {
      float a = os[i] * fac;
      for (int j = 0; j < cnt; ++j) a = fmaf(sc[j], F32In<DT>::ld(vp[((size_t)rows[j] * p.G + g) * p.Vp + i]), a);
      os[i] = a;
    }
  }
  float inv = p.score_bias != nullptr ? 1.0f : l_run > 0.f ? 1.0f / l_run : 0.f;
  if (p.sinks != nullptr && l_run > 0.f) {
    const float sink = p.sinks[h], mx = fmaxf(m_run, sink), fac = expf(m_run - mx);
    inv = fac / (l_run * fac + expf(sink - mx));
  }
  if (p.head_gate != nullptr) inv *= 1.0f / (1.0f + expf(-p.head_gate[(size_t)t * p.ld_head_gate + h]));
  T* op = reinterpret_cast<T*>(p.out) + (size_t)t * p.ld_out + (size_t)h * p.Vp;
  const T* gp = p.gate != nullptr ? reinterpret_cast<const T*>(p.gate) + (size_t)t * p.ld_gate + (size_t)h * p.Vp : nullptr;
  if (p.rot_v > 0) {
    const int at = pos < 0 ? 0 : pos >= p.tab_rows ? p.tab_rows - 1 : pos, half = p.rot_v >> 1;
    __syncthreads();
    for (int m = tid; m < half; m += 128) {
      const float c = p.cos_v[(size_t)at * half + m], s = p.sin_v[(size_t)at * half + m], u = os[2 * m], v = os[2 * m + 1];
      os[2 * m] = u * c + v * s;
      os[2 * m + 1] = v * c - u * s;
    }
    __syncthreads();
  }
  for (int i = tid; i < p.Vp; i += 128) {
    float v = os[i] * inv;
    if (gp != nullptr) v *= 1.0f / (1.0f + expf(-F32In<DT>::ld(gp[i])));
    op[i] = F32In<DT>::st(v);
  }
}

}  // namespace fb

using namespace fb;

// dt: 0 fp16, 1 bf16, 2 fp32 operands.  batch > 1: see Full32Params.  counts / offsets (optional): grouped rows, `batch` experts whose
// weights are batch_w_rows rows apart; max_rows bounds an expert's rows.
extern "C" int fb_gemm_full32(const void* X, const void* W, void* out, const void* bias, const float* residual, const void* gate, int M,
                              int N, int K, int batch, long long ldx, long long ldw, long long ld_out, long long ld_res, long long ld_gate,
                              long long batch_w_rows, long long batch_x_cols, long long batch_out_cols, const int* counts,
                              const int* offsets, float alpha, int act, int out_f32, const float* row_gate, long long ld_row_gate,
                              const void* mul, const int* mul_rows, long long ld_mul, int mul_count, int dt, void* stream) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  if (K <= 0 || dt < 0 || dt > 2 || batch > 65535 || act < 0 || act > 3 || (mul != nullptr && (mul_rows == nullptr || mul_count <= 0))) return -1;
  Full32Params p{X, W, out, residual, gate, bias, M, N, K, ldx, ldw, ld_out, ld_res, ld_gate, batch_w_rows, batch_x_cols, batch_out_cols,
                 counts, offsets, alpha, act, out_f32, row_gate, ld_row_gate, mul, mul_rows, ld_mul, mul_count};
  int gy = (M + 63) / 64;
  if (counts != nullptr && gy > 8) gy = 8;            // an expert rarely gets more; the kernel strides over the rest
  if (gy > 65535) gy = 65535;
  const dim3 grid((N + 63) / 64, gy, batch);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (dt == 0) gemm_full32_kernel<0><<<grid, 256, 0, s>>>(p);
  else if (dt == 1) gemm_full32_kernel<1><<<grid, 256, 0, s>>>(p);
  else gemm_full32_kernel<2><<<grid, 256, 0, s>>>(p);
  return (int)cudaGetLastError();
}

// q: [T, H, ld], pool: [num_slots, ld]; scores over the first R <= ld columns; out: [T, H, RV], the first RV <= R.  page_table [T, max_pages] and kv_lens [T] belong to the rows: row t
// sees keys [max(0, kv_lens[t] - window), kv_lens[t]).
extern "C" int fb_latent_attn32(const void* q, const void* pool, void* out, const int* page_table, const int* kv_lens, int T, int H, int R, int RV,
                                int ld, int max_pages, int page_len, int window, float scale, const float* head_gate, int dt, void* stream) {
  if (T <= 0 || H <= 0) return 0;
  if (R <= 0 || RV <= 0 || RV > R || ld < R || R > 24576 || H > 65535 || max_pages <= 0 || page_len <= 0 || dt < 0 || dt > 2) return -1;
  const size_t smem = (size_t)(R + RV) * 4;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define GO(DT)                                                                                                                     \
  {                                                                                                                                \
    static DeviceOnce cfg;                                                                                                         \
    if (cfg.need()) cudaFuncSetAttribute(latent_attn32_kernel<DT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 24576 * 8);         \
    latent_attn32_kernel<DT><<<dim3(T, H), 128, smem, s>>>((const F32In<DT>::T*)q, (const F32In<DT>::T*)pool, (F32In<DT>::T*)out,  \
                                                           page_table, kv_lens, max_pages, page_len, H, R, RV, ld, window, scale, head_gate); \
  }
  if (dt == 0) GO(0) else if (dt == 1) GO(1) else GO(2)
#undef GO
  return (int)cudaGetLastError();
}

// See Grouped32Params; q / out / gate: T rows, pools [num_pages * page_len, G, Dp / Vp].
extern "C" int fb_grouped_attn32(const void* q, long long ld_q, const void* k_pool, const void* v_pool, void* out, long long ld_out,
                                 const void* gate, long long ld_gate, const int* page_table, const int* kv_lens, int T, int H, int G, int D,
                                 int Dp, int Vp, int max_pages, int num_pages, int page_len, int window, int chunk, int keep, float scale,
                                 float softcap, const float* sinks, const float* head_gate, long long ld_head_gate, const float* score_bias, const float* cos_v,
                                 const float* sin_v, int rot_v, int tab_rows, int dt, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G != 0 || H > 65535 || D <= 0 || Dp < D || Vp <= 0 || Dp + Vp > 49152 || max_pages <= 0 || num_pages <= 0 ||
      page_len <= 0 || window < 0 || chunk < 0 || keep < 0 || dt < 0 || dt > 2 || rot_v < 0 || (rot_v & 1) || rot_v > Vp ||
      (rot_v > 0 && (cos_v == nullptr || sin_v == nullptr || tab_rows <= 0)))
    return -1;
  Grouped32Params p{q, k_pool, v_pool, out, gate, ld_q, ld_out, ld_gate, page_table, kv_lens, H, G, D, Dp, Vp, max_pages, num_pages, page_len, window, chunk, keep, scale, softcap, sinks, head_gate, ld_head_gate, score_bias, cos_v, sin_v, rot_v, tab_rows};
  const size_t smem = (size_t)(Dp + Vp) * 4;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define GO(DT)                                                                                                          \
  {                                                                                                                     \
    static DeviceOnce cfg;                                                                                              \
    if (cfg.need()) cudaFuncSetAttribute(grouped_attn32_kernel<DT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 49152 * 4); \
    grouped_attn32_kernel<DT><<<dim3(T, H), 128, smem, s>>>(p);                                                         \
  }
  if (dt == 0) GO(0) else if (dt == 1) GO(1) else GO(2)
#undef GO
  return (int)cudaGetLastError();
}
