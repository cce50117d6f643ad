// Real-gated linear recurrent unit (Griffin's recurrent block) for sm_100a.  Per channel, with u the output of a short causal convolution
// and r, i the sigmoids of two block-diagonal products of u:
//     log a = r * decay,   S_t = a S_(t-1) + sqrt(1 - a^2) i u,   out = S_t * gelu(y)           decay = -8 softplus(lam)
// The state S is fp32; beside it a request carries the convolution's last taps - 1 inputs, in the activation type.
//
//  * rglru_conv_kernel: u for all tokens; a thread slides over up to eight tokens of four channels.
//  * (the gates' logits are a block-diagonal tensor-core product, gemm_bf16.cu)
//  * rglru_sum_kernel: prompts of several chunks only: each chunk's product of decays (as a sum of logarithms) and what it adds to the state.
//  * rglru_scan_kernel: a chunk's state from the sums before it, its tokens, the output gate, the new states.  A request of one chunk
//    (a decoded token among them) needs this kernel alone.
// All chunks and channels run in parallel; a chunk adds up the sums of the chunks before it by itself.  State is read and written by
// different CTAs of a long request, so the first chunk's initial state travels through the sums' scratch.
//
// Compiled without fast-math: exponentials, square roots and divisions are the accurate ones.
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

constexpr int RG_CHUNK = 128;                      // most tokens of a chunk

struct RglruParams {
  const void* x; const void* y; long long ld;      // [T, ld] rows: the convolution's input, the output gate's
  const float* conv_w; const float* conv_b;        // [taps, W], [W]
  const float* gate_b;                             // [blocks, 2, part]: biases of r, then of i
  const float* decay;                              // [W] = -8 softplus(lam)
  const float* z;                                  // [T, 2 W]: a block's logits are [r part | i part]
  void* u;                                         // [T, W]
  void* out; long long ld_out;
  void* conv_state; float* state;                  // [slots, W, taps - 1], [slots, W]
  const int* slots;                                // one token per request: its slot (chunks null)
  // [n_chunks][6] = (first row, rows, slot, rows of the request before it in this batch, first chunk of the request, 1 if its last)
  const int* chunks;
  float* sum_a; float* sum_s; float* init;         // [n_chunks, W] sums of log a, state added; [n_chunks, W] (the first chunk's row): initial state
  int W, part, taps, n_chunks;
};

__device__ __forceinline__ void rg_chunk(const RglruParams& p, int c, int& row0, int& n, int& slot, int& before, int& first, bool& last) {
  if (p.chunks == nullptr) { row0 = c; n = 1; slot = p.slots[c]; before = 0; first = c; last = true; return; }
  const int* m = p.chunks + 6 * c;
  row0 = m[0]; n = m[1]; slot = m[2]; before = m[3]; first = m[4]; last = m[5] != 0;
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

// grid (chunks, ceil(W / 128), ceil(rows / 64)), 256 threads: 32 lanes of four channels x 8 groups of eight tokens.  KT: the taps (0: any)
template <int DT, int KT>
__global__ void __launch_bounds__(256) rglru_conv_kernel(const RglruParams p) {
  typedef typename RAct<DT>::T T;
  pdl_launch_dependents();
  pdl_wait();
  int row0, n, slot, before, first;
  bool last;
  rg_chunk(p, blockIdx.x, row0, n, slot, before, first, last);
  const int c = (blockIdx.y * 32 + (threadIdx.x & 31)) * 4, t0 = (blockIdx.z * 8 + (threadIdx.x >> 5)) * 8;
  if (c >= p.W || t0 >= n) return;
  const int K = KT > 0 ? KT : p.taps;
  const T* x = reinterpret_cast<const T*>(p.x);
  // input `back` tokens before token t of the chunk
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
    float w[KT > 0 ? KT : 1][4], win[KT > 0 ? KT : 1][4];
#pragma unroll
    for (int k = 0; k < KT; ++k) rg_ld4<2>(p.conv_w + (size_t)k * p.W + c, w[k]);
#pragma unroll
    for (int k = 1; k < KT; ++k) input(t0, KT - k, win[k]);
    for (int t = t0; t < t1; ++t) {
#pragma unroll
      for (int k = 0; k + 1 < KT; ++k)
#pragma unroll
        for (int j = 0; j < 4; ++j) win[k][j] = win[k + 1][j];
      input(t, 0, win[KT - 1]);
      float o[4] = {b[0], b[1], b[2], b[3]};
#pragma unroll
      for (int k = 0; k < KT; ++k)
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] = fmaf(w[k][j], win[k][j], o[j]);
      rg_st4<DT>(reinterpret_cast<T*>(p.u) + (size_t)(row0 + t) * p.W + c, o);
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

// log a of one token and channel, and what the token adds to the state
struct RgGates { float rb, ib, decay; int zc, zi; };
__device__ __forceinline__ RgGates rg_gates(const RglruParams& p, int c) {
  RgGates g;
  const int blk = c / p.part, j = c - blk * p.part;
  g.zc = 2 * blk * p.part + j;
  g.zi = g.zc + p.part;
  g.rb = p.gate_b[g.zc]; g.ib = p.gate_b[g.zi]; g.decay = p.decay[c];
  return g;
}
__device__ __forceinline__ void rg_step(const RgGates& g, float zr, float zi, float u, float& log_a, float& add) {
  log_a = g.decay / (1.0f + expf(-(zr + g.rb)));
  add = sqrtf(-expm1f(2.0f * log_a)) * u / (1.0f + expf(-(zi + g.ib)));
}

// grid (chunks, ceil(W / 128)), 128 threads: a channel each
template <int DT>
__global__ void __launch_bounds__(128) rglru_sum_kernel(const RglruParams p) {
  pdl_launch_dependents();
  pdl_wait();
  int row0, n, slot, before, first;
  bool last;
  rg_chunk(p, blockIdx.x, row0, n, slot, before, first, last);
  const int c = blockIdx.y * 128 + threadIdx.x;
  if (c >= p.W || (last && (int)blockIdx.x == first)) return;        // (a request of one chunk)
  float S = 0.f, la = 0.f;
  if ((int)blockIdx.x == first) {
    S = p.state[(size_t)slot * p.W + c];
    p.init[(size_t)first * p.W + c] = S;
  }
  if (last) return;                                                   // nothing follows it
  const RgGates g = rg_gates(p, c);
  const float* z = p.z + (size_t)row0 * 2 * p.W;
  const typename RAct<DT>::T* u = reinterpret_cast<const typename RAct<DT>::T*>(p.u) + (size_t)row0 * p.W + c;
#pragma unroll 8
  for (int t = 0; t < n; ++t) {
    float l, add;
    rg_step(g, z[(size_t)t * 2 * p.W + g.zc], z[(size_t)t * 2 * p.W + g.zi], RAct<DT>::ld(u[(size_t)t * p.W]), l, add);
    S = fmaf(expf(l), S, add);
    la += l;
  }
  p.sum_a[(size_t)blockIdx.x * p.W + c] = la;
  p.sum_s[(size_t)blockIdx.x * p.W + c] = S;                          // (the first chunk's includes the initial state)
}

template <int DT>
__global__ void __launch_bounds__(128) rglru_scan_kernel(const RglruParams p) {
  typedef typename RAct<DT>::T T;
  pdl_launch_dependents();
  pdl_wait();
  int row0, n, slot, before, first;
  bool last;
  rg_chunk(p, blockIdx.x, row0, n, slot, before, first, last);
  const int c = blockIdx.y * 128 + threadIdx.x;
  if (c >= p.W) return;
  float* state = p.state + (size_t)slot * p.W + c;
  const int me = blockIdx.x;
  float S;
  if (me == first) {
    S = last ? *state : p.init[(size_t)first * p.W + c];
  } else {
    S = p.sum_s[(size_t)first * p.W + c];
#pragma unroll 4
    for (int j = first + 1; j < me; ++j) S = fmaf(expf(p.sum_a[(size_t)j * p.W + c]), S, p.sum_s[(size_t)j * p.W + c]);
  }
  const RgGates g = rg_gates(p, c);
  const float* z = p.z + (size_t)row0 * 2 * p.W;
  const T* u = reinterpret_cast<const T*>(p.u) + (size_t)row0 * p.W + c;
  const T* y = reinterpret_cast<const T*>(p.y) + (size_t)row0 * p.ld + c;
  T* out = reinterpret_cast<T*>(p.out) + (size_t)row0 * p.ld_out + c;
#pragma unroll 8
  for (int t = 0; t < n; ++t) {
    float l, add;
    rg_step(g, z[(size_t)t * 2 * p.W + g.zc], z[(size_t)t * 2 * p.W + g.zi], RAct<DT>::ld(u[(size_t)t * p.W]), l, add);
    S = fmaf(expf(l), S, add);
    const float v = RAct<DT>::ld(y[(size_t)t * p.ld]);
    out[(size_t)t * p.ld_out] = RAct<DT>::st(S * 0.5f * v * (1.0f + tanhf(0.79788456080286536f * (v + 0.044715f * v * v * v))));
  }
  if (!last) return;
  *state = S;
  // the last taps - 1 inputs of [what the state held | the request's rows of this batch]; ascending, so that old entries are read first
  const int K1 = p.taps - 1, rows = before + n;
  T* cs = reinterpret_cast<T*>(p.conv_state) + ((size_t)slot * p.W + c) * K1;
  const T* x = reinterpret_cast<const T*>(p.x) + (size_t)(row0 - before) * p.ld + c;
  for (int j = 0; j < K1; ++j) {
    const int at = rows + j - K1;
    cs[j] = at >= 0 ? x[(size_t)at * p.ld] : cs[rows + j];
  }
}

}  // namespace fb

using namespace fb;

// One block: everything between the input projections, with the gates' logits computed by the caller in between: step 0 is the convolution,
// step 1 the recurrence.  x / y: [T, ld] (columns of the projection), u [T, W], z [T, 2 W], out [T, >= W].  chunks (n_chunks of at most
// 128 rows) or, for one token per request, slots [n_chunks].  multi: some request has several chunks (sum_a, sum_s, init: [n_chunks, W]).
// W a multiple of 8, `part` channels a block; see RglruParams.  dt: 0 fp16, 1 bf16, 2 fp32.
extern "C" int fb_rglru(int step, const void* x, const void* y, long long ld, const float* conv_w, const float* conv_b, const float* gate_b, const float* decay,
                        const float* z, void* u, void* out, long long ld_out, void* conv_state, float* state, const int* slots, const int* chunks,
                        int n_chunks, int max_rows, int multi, float* sum_a, float* sum_s, float* init, int W, int part, int taps, int dt, void* stream) {
  if (n_chunks <= 0) return 0;
  if (W <= 0 || W % 8 != 0 || part <= 0 || W % part != 0 || taps <= 0 || dt < 0 || dt > 2 || max_rows <= 0 || max_rows > RG_CHUNK || ld % 8 != 0 || (reinterpret_cast<uintptr_t>(x) & 15) ||
      (chunks == nullptr && (slots == nullptr || multi || max_rows != 1)) || (multi && (sum_a == nullptr || sum_s == nullptr || init == nullptr)))
    return -1;
  RglruParams p{x, y, ld, conv_w, conv_b, gate_b, decay, z, u, out, ld_out, conv_state, state, slots, chunks, sum_a, sum_s, init, W, part, taps, n_chunks};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const dim3 lanes((unsigned)n_chunks, (unsigned)((W + 127) / 128));
  if (step == 0) {
    const dim3 grid(lanes.x, lanes.y, (unsigned)((max_rows + 63) / 64));
#define GO(DT, K) launch_k(rglru_conv_kernel<DT, K>, grid, dim3(256), 0, s, 0, p)
#define GO_K(DT) { if (taps == 2) GO(DT, 2); else if (taps == 3) GO(DT, 3); else if (taps == 4) GO(DT, 4); else GO(DT, 0); }
    if (dt == 0) GO_K(0) else if (dt == 1) GO_K(1) else GO_K(2)
#undef GO_K
#undef GO
  } else {
#define GO(KERN) { if (dt == 0) launch_k(KERN<0>, lanes, dim3(128), 0, s, 0, p); else if (dt == 1) launch_k(KERN<1>, lanes, dim3(128), 0, s, 0, p); else launch_k(KERN<2>, lanes, dim3(128), 0, s, 0, p); }
    if (multi) GO(rglru_sum_kernel)
    GO(rglru_scan_kernel)
#undef GO
  }
  return (int)cudaGetLastError();
}
