// Real-gated linear recurrent unit (Griffin's recurrent block) for sm_100a.  Per channel, with u the output of a short causal convolution
// and r, i the sigmoids of two block-diagonal products of u:
//     log a = r * decay,   S_t = a S_(t-1) + sqrt(1 - a^2) i u,   out = S_t * gelu(y)           decay = -8 softplus(lam)
// The state S is fp32; beside it a request carries the convolution's last taps - 1 inputs, in the activation type.
//
//  * rglru_conv_kernel: u for all tokens; a thread takes up to eight tokens of four channels.
//  * (the gates' logits are a block-diagonal tensor-core product, gemm_bf16.cu)
//  * rglru_step_kernel: short requests (decoded tokens among them); a thread walks one channel.
//  * longer portions in chunks of 128 tokens that run in parallel; a thread walks one channel of a chunk, the next tokens' operands on their way:
//      rglru_sum_kernel    a chunk's sum of log a and the state it ends with (from zero; the request's first chunk from its state)
//      rglru_scan_kernel   composes the sums of the chunks before it, then its own tokens, the output gate and the new states
//    State is read and written by different CTAs of a request, so its initial state travels through the sums' scratch.
// 1 - a^2 = -m (2 + m) with m = e^(log a) - 1, so that channels that hardly forget lose nothing to cancellation.  Compiled without
// fast-math; float32 models take the accurate functions, 16-bit ones the special-function unit's (a few units in the last fp32 place).
#include "ptx.cuh"
#include "launch.h"

FB_DEFINE_ERROR_API(rglru)

namespace fb {

template <int DT> struct RAct;
template <> struct RAct<0> { typedef uint16_t T; static __device__ __forceinline__ float ld(uint16_t v) { return __half2float(__ushort_as_half(v)); }
                             static __device__ __forceinline__ uint16_t st(float v) { return __half_as_ushort(__float2half_rn(v)); } };
template <> struct RAct<1> { typedef uint16_t T; static __device__ __forceinline__ float ld(uint16_t v) { return __bfloat162float(__ushort_as_bfloat16(v)); }
                             static __device__ __forceinline__ uint16_t st(float v) { return __bfloat16_as_ushort(__float2bfloat16_rn(v)); } };
template <> struct RAct<2> { typedef float T; static __device__ __forceinline__ float ld(float v) { return v; } static __device__ __forceinline__ float st(float v) { return v; } };

constexpr int RG_CHUNK = 128;                      // most tokens of an item

struct RglruParams {
  const void* x; const void* y; long long ld;      // [T, ld] rows: the convolution's input, the output gate's
  const float* conv_w; const float* conv_b;        // [taps, W], [W]
  const float* gate_b;                             // [blocks, 2, part]: biases of r, then of i
  const float* decay;                              // [W] = -8 softplus(lam)
  const float* z;                                  // [T, 2 W]: a block's logits are [r part | i part]
  void* u;                                         // [T, W]
  void* out; long long ld_out;
  void* conv_state; float* state;                  // [slots, W, taps - 1], [slots, W]
  const int* slots;                                // one token per request: its slot (items null)
  // [items][6] = (first row, rows, slot, rows of the request before these in this batch, the request's first item, 1 if its last)
  const int* items;
  float* sum_a; float* sum_s; float* init;         // [items, W]: sums of log a, states; the request's initial state (its first item's row)
  int W, part, taps;
};

__device__ __forceinline__ void rg_item(const RglruParams& p, int i, int& row0, int& n, int& slot, int& before) {
  if (p.items == nullptr) { row0 = i; n = 1; slot = p.slots[i]; before = 0; return; }
  const int* m = p.items + 6 * i;
  row0 = m[0]; n = m[1]; slot = m[2]; before = m[3];
}

template <int DT>
__device__ __forceinline__ void rg_ld4(const typename RAct<DT>::T* p, float* v) {
  if (DT == 2) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  } else {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_16<DT == 1>(t.x), b = unpack_16<DT == 1>(t.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
}
template <int DT>
__device__ __forceinline__ void rg_st4(typename RAct<DT>::T* p, const float* v) {
  if (DT == 2) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *reinterpret_cast<uint2*>(p) = make_uint2(pack_16<DT == 1>(v[0], v[1]), pack_16<DT == 1>(v[2], v[3]));
}

// grid (items, ceil(W / 128), ceil(rows / 64)), 256 threads: 32 lanes of four channels x 8 groups of eight tokens.  KT: the taps (0: any)
template <int DT, int KT>
__global__ void __launch_bounds__(256) rglru_conv_kernel(const RglruParams p) {
  typedef typename RAct<DT>::T T;
  pdl_launch_dependents();
  pdl_wait();
  int row0, n, slot, before;
  rg_item(p, blockIdx.x, row0, n, slot, before);
  const int c = (blockIdx.y * 32 + (threadIdx.x & 31)) * 4, t0 = (blockIdx.z * 8 + (threadIdx.x >> 5)) * 8;
  if (c >= p.W || t0 >= n) return;
  const int K = KT > 0 ? KT : p.taps;
  const T* x = reinterpret_cast<const T*>(p.x);
  // input `back` tokens before token t of the item
  auto input = [&](int t, int back, float* v) {
    const int at = before + t - back;                      // place within the request's rows of this batch
    if (at >= 0) { rg_ld4<DT>(x + (size_t)(row0 + t - back) * p.ld + c, v); return; }
    const T* st = reinterpret_cast<const T*>(p.conv_state) + ((size_t)slot * p.W + c) * (K - 1) + (K - 1 + at);
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = RAct<DT>::ld(st[(size_t)j * (K - 1)]);
  };
  float b[4];
  rg_ld4<2>(p.conv_b + c, b);
  const int t1 = min(t0 + 8, n);
  if (KT > 0) {
    // all inputs are requested before the first is used: the KT - 1 before the tokens, then theirs
    float w[KT > 0 ? KT : 1][4], in[8 + (KT > 0 ? KT - 1 : 0)][4];
    if (before + t0 >= KT - 1) {
      const T* xp = x + (size_t)(row0 + t0 - (KT - 1)) * p.ld + c;
#pragma unroll
      for (int i = 0; i < 8 + KT - 1; ++i)
        if (t0 + i - (KT - 1) < t1) rg_ld4<DT>(xp + (size_t)i * p.ld, in[i]);
    } else {
#pragma unroll
      for (int i = 0; i < 8 + KT - 1; ++i)
        if (t0 + i - (KT - 1) < t1) input(t0 + i, KT - 1, in[i]);
    }
#pragma unroll
    for (int k = 0; k < KT; ++k) rg_ld4<2>(p.conv_w + (size_t)k * p.W + c, w[k]);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (t0 + i >= t1) break;
      float o[4] = {b[0], b[1], b[2], b[3]};
#pragma unroll
      for (int k = 0; k < KT; ++k)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] = fmaf(w[k][j], in[i + k][j], o[j]);
      rg_st4<DT>(reinterpret_cast<T*>(p.u) + (size_t)(row0 + t0 + i) * p.W + c, o);
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float o[4] = {b[0], b[1], b[2], b[3]}, w[4], v[4];
      for (int k = 0; k < K; ++k) {
        rg_ld4<2>(p.conv_w + (size_t)k * p.W + c, w);
        input(t, K - 1 - k, v);
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] = fmaf(w[j], v[j], o[j]);
      }
      rg_st4<DT>(reinterpret_cast<T*>(p.u) + (size_t)(row0 + t) * p.W + c, o);
    }
  }
}

struct RgGates { float rb, ib, decay; int zc, zi; };
__device__ __forceinline__ RgGates rg_gates(const RglruParams& p, int c) {
  RgGates g;
  const int blk = c / p.part, j = c - blk * p.part;
  g.zc = 2 * blk * p.part + j;
  g.zi = g.zc + p.part;
  g.rb = p.gate_b[g.zc]; g.ib = p.gate_b[g.zi]; g.decay = p.decay[c];
  return g;
}
// the special-function unit's operations, denormals flushed
__device__ __forceinline__ float rg_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float rg_rcp(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float rg_sqrt(float x) { float y; asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
constexpr float RG_LOG2E = 1.4426950408889634f;

// e^x - 1, x <= 0: the Taylor polynomial of degree 7 near zero (its next term is below 3e-8 of the sum), the exponential elsewhere
__device__ __forceinline__ float rg_expm1(float x) {
  float y = fmaf(x, 1.f / 5040.f, 1.f / 720.f);
  y = fmaf(x, y, 1.f / 120.f);
  y = fmaf(x, y, 1.f / 24.f);
  y = fmaf(x, y, 1.f / 6.f);
  y = fmaf(x, y, 0.5f);
  y = fmaf(x * x, y, x);
  return x > -0.35f ? y : rg_ex2(x * RG_LOG2E) - 1.f;
}
template <bool EXACT>
__device__ __forceinline__ float rg_sigmoid(float z) {
  return EXACT ? 1.0f / (1.0f + expf(-z)) : rg_rcp(1.0f + rg_ex2(-RG_LOG2E * z));
}
// decay, its logarithm and what the token adds
template <bool EXACT>
__device__ __forceinline__ void rg_step(const RgGates& g, float zr, float zi, float u, float& log_a, float& a, float& add) {
  log_a = g.decay * rg_sigmoid<EXACT>(zr + g.rb);
  const float m = EXACT ? expm1f(log_a) : rg_expm1(log_a), v = -m * (2.0f + m);
  a = 1.0f + m;
  add = (EXACT ? sqrtf(v) : rg_sqrt(v)) * u * rg_sigmoid<EXACT>(zi + g.ib);
}

template <bool EXACT>
__device__ __forceinline__ float rg_gelu(float v) {                       // (1 + tanh w) / 2 = sigmoid(2 w)
  const float w = 0.79788456080286536f * (v + 0.044715f * v * v * v);
  return v * (EXACT ? 0.5f * (1.0f + tanhf(w)) : rg_sigmoid<false>(2.0f * w));
}

// The last taps - 1 inputs of [what the state held | the request's n rows]; ascending, so that old entries are read before they are replaced
template <int DT>
__device__ __forceinline__ void rg_keep_inputs(const RglruParams& p, int c, int row0, int n, int slot) {
  typedef typename RAct<DT>::T T;
  const int K1 = p.taps - 1;
  T* cs = reinterpret_cast<T*>(p.conv_state) + ((size_t)slot * p.W + c) * K1;
  const T* x = reinterpret_cast<const T*>(p.x) + (size_t)row0 * p.ld + c;
  for (int j = 0; j < K1; ++j) {
    const int at = n + j - K1;
    cs[j] = at >= 0 ? x[(size_t)at * p.ld] : cs[n + j];
  }
}

// grid (items, ceil(W / 128)), 128 threads: a channel each
template <int DT>
__global__ void __launch_bounds__(128) rglru_step_kernel(const RglruParams p) {
  typedef typename RAct<DT>::T T;
  pdl_launch_dependents();
  pdl_wait();
  int row0, n, slot, before;
  rg_item(p, blockIdx.x, row0, n, slot, before);
  const int c = blockIdx.y * 128 + threadIdx.x;
  if (c >= p.W || n <= 0) return;
  float* state = p.state + (size_t)slot * p.W + c;
  float S = *state;
  const RgGates g = rg_gates(p, c);
  const float* z = p.z + (size_t)row0 * 2 * p.W;
  const T* u = reinterpret_cast<const T*>(p.u) + (size_t)row0 * p.W + c;
  const T* y = reinterpret_cast<const T*>(p.y) + (size_t)row0 * p.ld + c;
  T* out = reinterpret_cast<T*>(p.out) + (size_t)row0 * p.ld_out + c;
  for (int t = 0; t < n; ++t) {
    float l, a, add;
    rg_step<DT == 2>(g, __ldg(z + g.zc), __ldg(z + g.zi), RAct<DT>::ld(__ldg(u)), l, a, add);
    S = fmaf(a, S, add);
    *out = RAct<DT>::st(S * rg_gelu<DT == 2>(RAct<DT>::ld(__ldg(y))));
    z += 2 * p.W; u += p.W; y += p.ld; out += p.ld_out;
  }
  *state = S;
  rg_keep_inputs<DT>(p, c, row0, n, slot);
}

// One channel's tokens of a chunk.  each(t, log a, a, what it adds, gate input)
constexpr int RG_BATCH = 4;
template <int DT, bool GATED, class Each>
__device__ __forceinline__ void rg_walk(const RglruParams& p, int c, int row0, int n, const Each& each) {
  typedef typename RAct<DT>::T T;
  const RgGates g = rg_gates(p, c);
  const float* z = p.z + (size_t)row0 * 2 * p.W + g.zc;
  const T* u = reinterpret_cast<const T*>(p.u) + (size_t)row0 * p.W + c;
  const T* y = reinterpret_cast<const T*>(p.y) + (size_t)row0 * p.ld + c;
  float zr[RG_BATCH], zi[RG_BATCH];
  T uu[RG_BATCH], yy[RG_BATCH];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int j = 0; j < RG_BATCH; ++j) {
      if (t0 + j < n) {
        zr[j] = __ldg(z); zi[j] = __ldg(z + p.part); uu[j] = __ldg(u);
        if (GATED) yy[j] = __ldg(y);
        z += 2 * p.W; u += p.W; y += p.ld;
      }
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < n; t0 += RG_BATCH) {
    float r[RG_BATCH], i[RG_BATCH], uf[RG_BATCH], yf[RG_BATCH];
#pragma unroll
    for (int j = 0; j < RG_BATCH; ++j) { r[j] = zr[j]; i[j] = zi[j]; uf[j] = RAct<DT>::ld(uu[j]); yf[j] = GATED ? RAct<DT>::ld(yy[j]) : 0.f; }
    fetch(t0 + RG_BATCH);
#pragma unroll
    for (int j = 0; j < RG_BATCH; ++j) {
      if (t0 + j < n) {
        float l, a, add;
        rg_step<DT == 2>(g, r[j], i[j], uf[j], l, a, add);
        each(t0 + j, l, a, add, yf[j]);
      }
    }
  }
}

// grid (items, ceil(W / 128)), 128 threads: a channel each
template <int DT>
__global__ void __launch_bounds__(128) rglru_sum_kernel(const RglruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  int row0, n, slot, before;
  rg_item(p, blockIdx.x, row0, n, slot, before);
  const int me = blockIdx.x, c = blockIdx.y * 128 + threadIdx.x;
  const bool first = p.items[6 * me + 4] == me, last = p.items[6 * me + 5] != 0;
  if (c >= p.W || (first && last)) return;                             // (a request of one chunk needs no sums)
  const size_t at = (size_t)me * p.W + c;
  float S = 0.f, la = 0.f;
  if (first) p.init[at] = S = p.state[(size_t)slot * p.W + c];
  if (last) return;                                                     // nothing follows it
  rg_walk<DT, false>(p, c, row0, n, [&](int, float l, float a, float add, float) {
    S = fmaf(a, S, add);
    la += l;
  });
  p.sum_a[at] = la;
  p.sum_s[at] = S;
}

template <int DT>
__global__ void __launch_bounds__(128) rglru_scan_kernel(const RglruParams p) {
  typedef typename RAct<DT>::T T;
  pdl_launch_dependents();
  pdl_wait();
  int row0, n, slot, before;
  rg_item(p, blockIdx.x, row0, n, slot, before);
  const int me = blockIdx.x, c = blockIdx.y * 128 + threadIdx.x;
  if (c >= p.W || n <= 0) return;
  const int first = p.items[6 * me + 4];
  const bool last = p.items[6 * me + 5] != 0;
  float* state = p.state + (size_t)slot * p.W + c;
  float S;
  if (me == first) {
    S = last ? *state : p.init[(size_t)me * p.W + c];
  } else {
    constexpr int N = 8;
    S = __ldg(p.sum_s + (size_t)first * p.W + c);
    const float* sa = p.sum_a + (size_t)(first + 1) * p.W + c;
    const float* ss = p.sum_s + (size_t)(first + 1) * p.W + c;
    for (int j0 = first + 1; j0 < me; j0 += N, sa += (size_t)N * p.W, ss += (size_t)N * p.W) {
      float la[N], add[N];
#pragma unroll
      for (int j = 0; j < N; ++j)
        if (j0 + j < me) { la[j] = __ldg(sa + (size_t)j * p.W); add[j] = __ldg(ss + (size_t)j * p.W); }
#pragma unroll
      for (int j = 0; j < N; ++j)
        if (j0 + j < me) S = fmaf(DT == 2 ? expf(la[j]) : rg_ex2(la[j] * RG_LOG2E), S, add[j]);
    }
  }
  T* out = reinterpret_cast<T*>(p.out) + (size_t)row0 * p.ld_out + c;
  rg_walk<DT, true>(p, c, row0, n, [&](int t, float, float a, float add, float v) {
    S = fmaf(a, S, add);
    out[(size_t)t * p.ld_out] = RAct<DT>::st(S * rg_gelu<DT == 2>(v));
  });
  if (!last) return;
  *state = S;
  rg_keep_inputs<DT>(p, c, row0 - before, before + n, slot);
}

}  // namespace fb

using namespace fb;

// Everything between the input projections of a layer but for the gates' logits, which the caller computes between step 0, the convolution,
// and the recurrence.  x / y: [T, ld] (columns of the projection), u [T, W], z [T, 2 W], out [T, >= W].
// Step 0: items of at most 128 rows (max_rows).  Step 1: n_items whole requests, token by token; without items, one token per request,
// slots [n_items].  Step 2: items as in step 0; multi: some request has several (sum_a, sum_s, init [n_items, W]).
// W a multiple of 8, `part` (a multiple of 8) channels a block; see RglruParams.  dt: 0 fp16, 1 bf16, 2 fp32.
extern "C" int fb_rglru(int step, const void* x, const void* y, long long ld, const float* conv_w, const float* conv_b, const float* gate_b, const float* decay,
                        const float* z, void* u, void* out, long long ld_out, void* conv_state, float* state, const int* slots, const int* items,
                        int n_items, int max_rows, int multi, float* sum_a, float* sum_s, float* init, int W, int part, int taps, int dt, void* stream) {
  if (n_items <= 0) return 0;
  if (W <= 0 || part <= 0 || part % 8 != 0 || W % part != 0 || taps <= 0 || dt < 0 || dt > 2 || max_rows <= 0 || (step != 1 && max_rows > RG_CHUNK) || ld % 8 != 0 ||
      (reinterpret_cast<uintptr_t>(x) & 15) || (items == nullptr && (slots == nullptr || max_rows != 1 || step == 2)) ||
      (multi && (sum_a == nullptr || sum_s == nullptr || init == nullptr)))
    return -1;
  RglruParams p{x, y, ld, conv_w, conv_b, gate_b, decay, z, u, out, ld_out, conv_state, state, slots, items, sum_a, sum_s, init, W, part, taps};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
#define GO(KERN, GRID, THREADS)                                                       \
  {                                                                                   \
    if (dt == 0) launch_k(KERN<0>, GRID, dim3(THREADS), 0, s, 0, p);                  \
    else if (dt == 1) launch_k(KERN<1>, GRID, dim3(THREADS), 0, s, 0, p);             \
    else launch_k(KERN<2>, GRID, dim3(THREADS), 0, s, 0, p);                          \
  }
  if (step == 0) {
    const dim3 grid((unsigned)n_items, (unsigned)((W + 127) / 128), (unsigned)((max_rows + 63) / 64));
#define GO_C(DT, K) launch_k(rglru_conv_kernel<DT, K>, grid, dim3(256), 0, s, 0, p)
#define GO_K(DT) { if (taps == 2) GO_C(DT, 2); else if (taps == 3) GO_C(DT, 3); else if (taps == 4) GO_C(DT, 4); else GO_C(DT, 0); }
    if (dt == 0) GO_K(0) else if (dt == 1) GO_K(1) else GO_K(2)
#undef GO_K
#undef GO_C
  } else if (step == 1) {
    const dim3 grid((unsigned)n_items, (unsigned)((W + 127) / 128));
    GO(rglru_step_kernel, grid, 128)
  } else {
    const dim3 grid((unsigned)n_items, (unsigned)((W + 127) / 128));
    if (multi) GO(rglru_sum_kernel, grid, 128)
    GO(rglru_scan_kernel, grid, 128)
  }
#undef GO
  return (int)cudaGetLastError();
}
