// Operators of models whose residual stream is fp32: token embedding plus sinusoidal or learned positions, RMSNorm of an fp32 row
// into the activation type, latent rows (norms, rotary key part) into the cache, per-head norm + rotary + cache append, and the end of
// a sub-layer (output norm, residual, next norm) for a plain output or a mixture-of-experts combine, or of a layer whose sub-layers
// stand side by side behind gates of their own.
//
// One CTA owns a row; the row stays in shared memory between the reduction and the normalised write, so every operand is read
// once.  Compiled without fast-math: angles, square roots and divisions are the correctly rounded fp32 ones.
// Activation type codes: 0 fp16, 1 bf16, 2 fp32.
#include "ptx.cuh"
#include "launch.h"

FB_DEFINE_ERROR_API(stream32)

namespace fb {

template <int DT>
struct Act;
template <>
struct Act<0> {
  typedef uint16_t T;
  static __device__ __forceinline__ float ld(uint16_t v) { return __half2float(__ushort_as_half(v)); }
  static __device__ __forceinline__ uint16_t st(float v) { return __half_as_ushort(__float2half_rn(v)); }
};
template <>
struct Act<1> {
  typedef uint16_t T;
  static __device__ __forceinline__ float ld(uint16_t v) { return __bfloat162float(__ushort_as_bfloat16(v)); }
  static __device__ __forceinline__ uint16_t st(float v) { return __bfloat16_as_ushort(__float2bfloat16_rn(v)); }
};
template <>
struct Act<2> {
  typedef float T;
  static __device__ __forceinline__ float ld(float v) { return v; }
  static __device__ __forceinline__ float st(float v) { return v; }
};

// four consecutive elements; the vector forms need 4-element alignment, which the launchers check
template <int DT>
__device__ __forceinline__ void ld4(const typename Act<DT>::T* p, float* v) {
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
__device__ __forceinline__ void st4(typename Act<DT>::T* p, const float* v) {
  if (DT == 2) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_16<DT == 1>(v[0], v[1]), pack_16<DT == 1>(v[2], v[3]));
  }
}

__device__ __forceinline__ float block_sum32(float v, float* sh) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) t += sh[w];
  return t;
}

// y = row * inv * w from the shared-memory copy of the row
template <int DT, int VEC>
__device__ __forceinline__ void norm_write(const float* row, const typename Act<DT>::T* w, typename Act<DT>::T* y, int H, float inv) {
  if (VEC == 4) {
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
      float wv[4], o[4];
      ld4<DT>(w + i, wv);
      const float4 r = *reinterpret_cast<const float4*>(row + i);
      o[0] = r.x * inv * wv[0]; o[1] = r.y * inv * wv[1]; o[2] = r.z * inv * wv[2]; o[3] = r.w * inv * wv[3];
      st4<DT>(y + i, o);
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) y[i] = Act<DT>::st(row[i] * inv * Act<DT>::ld(w[i]));
  }
}

// the same, or the row itself where there is no weight
template <int DT, int VEC>
__device__ __forceinline__ void row_write(const float* row, const typename Act<DT>::T* w, typename Act<DT>::T* y, int H, float inv) {
  if (w != nullptr) { norm_write<DT, VEC>(row, w, y, H, inv); return; }
  for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {
    if (VEC == 4) st4<DT>(y + i, row + i); else y[i] = Act<DT>::st(row[i]);
  }
}

// y[row] = RMSNorm(x[row]) * w
template <int DT, int VEC>
__global__ void rmsnorm32_kernel(const float* __restrict__ x, const typename Act<DT>::T* __restrict__ w, typename Act<DT>::T* __restrict__ y,
                                 int H, int ldx, int ldy, float eps) {
  extern __shared__ float row[];
  __shared__ float sh[32];
  pdl_launch_dependents();
  pdl_wait();
  const float* xp = x + (size_t)blockIdx.x * ldx;
  float ss = 0.f;
  if (VEC == 4) {
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(xp + i);
      *reinterpret_cast<float4*>(row + i) = v;
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int i = threadIdx.x; i < H; i += blockDim.x) { const float v = xp[i]; row[i] = v; ss += v * v; }
  }
  ss = block_sum32(ss, sh);
  const float inv = 1.0f / sqrtf(ss / (float)H + eps);
  norm_write<DT, VEC>(row, w, y + (size_t)blockIdx.x * ldy, H, inv);
}

// h[t] = table[ids[t]] + position in fp32, and its RMSNorm (w == nullptr: the row itself; y == nullptr: h only).  inv_freq: the position
// is sines and cosines, inv_freq[i] = 10000^(-2i / H) in double; the angle is reduced to [-pi, pi] in double, so a far position costs
// no accuracy.  pos_table: it is row positions[t] of a learned table.  add_vec: one more row that every token gets.
template <int DT, int VEC>
__global__ void embed_pos_norm_kernel(const int* __restrict__ ids, const int* __restrict__ positions, const typename Act<DT>::T* __restrict__ table,
                                      const double* __restrict__ inv_freq, const typename Act<DT>::T* __restrict__ pos_table, int pos_rows,
                                      const typename Act<DT>::T* __restrict__ add_vec, const typename Act<DT>::T* __restrict__ w,
                                      float* __restrict__ h, typename Act<DT>::T* __restrict__ y, int H, int vocab, float eps) {
  extern __shared__ float row[];
  __shared__ float sh[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  int id = ids[t];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const typename Act<DT>::T* e = table + (size_t)id * H;
  float* hp = h + (size_t)t * H;
  int row_p = positions[t];
  const double pos = (double)row_p;
  row_p = row_p < 0 ? 0 : (row_p >= pos_rows ? pos_rows - 1 : row_p);
  const typename Act<DT>::T* pe = pos_table != nullptr ? pos_table + (size_t)row_p * H : nullptr;
  float ss = 0.f;
  auto add_pos = [&](int i, float& a, float& b) {
    const double ang = pos * inv_freq[i];
    const float red = (float)(ang - 6.283185307179586476925 * rint(ang * 0.15915494309189533577));
    float s, c;
    sincosf(red, &s, &c);
    a += s; b += c;
  };
  if (VEC == 4) {
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
      float v[4];
      ld4<DT>(e + i, v);
      if (inv_freq != nullptr) { add_pos(i / 2, v[0], v[1]); add_pos(i / 2 + 1, v[2], v[3]); }
      if (pe != nullptr) {
        float u[4];
        ld4<DT>(pe + i, u);
        v[0] += u[0]; v[1] += u[1]; v[2] += u[2]; v[3] += u[3];
      }
      if (add_vec != nullptr) {
        float u[4];
        ld4<DT>(add_vec + i, u);
        v[0] += u[0]; v[1] += u[1]; v[2] += u[2]; v[3] += u[3];
      }
      st4<2>(hp + i, v);
      st4<2>(row + i, v);
      ss += v[0] * v[0] + v[1] * v[1] + v[2] * v[2] + v[3] * v[3];
    }
  } else {
    for (int i = threadIdx.x; 2 * i < H; i += blockDim.x) {
      const bool two = 2 * i + 1 < H;
      float a = Act<DT>::ld(e[2 * i]), b = two ? Act<DT>::ld(e[2 * i + 1]) : 0.f;
      if (inv_freq != nullptr) add_pos(i, a, b);
      if (pe != nullptr) { a += Act<DT>::ld(pe[2 * i]); if (two) b += Act<DT>::ld(pe[2 * i + 1]); }
      if (add_vec != nullptr) { a += Act<DT>::ld(add_vec[2 * i]); if (two) b += Act<DT>::ld(add_vec[2 * i + 1]); }
      hp[2 * i] = a; row[2 * i] = a; ss += a * a;
      if (two) { hp[2 * i + 1] = b; row[2 * i + 1] = b; ss += b * b; }
    }
  }
  if (y == nullptr) return;
  ss = block_sum32(ss, sh);
  const float inv = 1.0f / sqrtf(ss / (float)H + eps);
  row_write<DT, VEC>(row, w, y + (size_t)t * H, H, inv);
}

// Everything between the input projection of latent attention and its next product, one CTA per token:
//   cq[t] = RMSNorm(query latent) * q_norm                              (q_rank > 0; columns [q_rank, q_pad) are zero)
//   pool[slot] = [RMSNorm(latent) * kv_norm | 0 | rotated key part | 0]  (rank of lv columns, rot of ld - lv; slots < 0 go to `spare`)
//   gates[t] = the head gates' logits in fp32                            (n_gates > 0)
struct LatentPostParams {
  const void* x; long long ldx;
  int q_col, q_rank, q_pad, kv_col, rank, lv, rot_col, rot, ld, neox, gate_col, n_gates;
  const void* q_norm; const void* kv_norm;
  const float* cos_tab; const float* sin_tab;
  int tab_rows;
  const int* positions; const int* slots;
  void* cq; void* pool; float* gates;
  long long spare;
  float eps;
};

template <int DT, int VEC>
__device__ __forceinline__ void ldv(const typename Act<DT>::T* p, float* v) {
  if (VEC == 4) ld4<DT>(p, v); else v[0] = Act<DT>::ld(p[0]);
}
template <int DT, int VEC>
__device__ __forceinline__ void stv(typename Act<DT>::T* p, const float* v) {
  if (VEC == 4) st4<DT>(p, v); else p[0] = Act<DT>::st(v[0]);
}

template <int DT, int VEC>
__global__ void latent_post_kernel(const LatentPostParams p) {
  typedef typename Act<DT>::T T;
  extern __shared__ float row[];
  __shared__ float sh[2][32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const T* xp = reinterpret_cast<const T*>(p.x) + (size_t)t * p.ldx;
  const int slot = p.slots[t];
  T* yp = reinterpret_cast<T*>(p.pool) + (size_t)(slot < 0 ? p.spare : (long long)slot) * p.ld;
  float sum[2] = {0.f, 0.f};
  float* krow = row + p.q_rank;
  auto take = [&](const T* src, float* dst, int n, float& s) {
    for (int i = threadIdx.x * VEC; i < n; i += blockDim.x * VEC) {
      float v[VEC];
      ldv<DT, VEC>(src + i, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) { dst[i + j] = v[j]; s += v[j] * v[j]; }
    }
  };
  take(xp + p.q_col, row, p.q_rank, sum[0]);
  take(xp + p.kv_col, krow, p.rank, sum[1]);
  for (int i = threadIdx.x; i < p.n_gates; i += blockDim.x) p.gates[(size_t)t * p.n_gates + i] = Act<DT>::ld(xp[p.gate_col + i]);
  if (p.rot > 0) {
    int pos = p.positions[t];
    pos = pos < 0 ? 0 : (pos >= p.tab_rows ? p.tab_rows - 1 : pos);
    const int half = p.rot >> 1;
    for (int j = threadIdx.x; 2 * j < p.ld - p.lv; j += blockDim.x) {
      if (j < half) {
        const int i0 = p.neox ? j : 2 * j, i1 = p.neox ? j + half : 2 * j + 1;
        const float c = p.cos_tab[(size_t)pos * half + j], s = p.sin_tab[(size_t)pos * half + j];
        const float u = Act<DT>::ld(xp[p.rot_col + i0]), v = Act<DT>::ld(xp[p.rot_col + i1]);
        yp[p.lv + i0] = Act<DT>::st(u * c - v * s);
        yp[p.lv + i1] = Act<DT>::st(v * c + u * s);
      } else {
        yp[p.lv + 2 * j] = yp[p.lv + 2 * j + 1] = Act<DT>::st(0.f);
      }
    }
  }
  // both sums in one exchange
#pragma unroll
  for (int k = 0; k < 2; ++k) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum[k] += __shfl_xor_sync(0xffffffffu, sum[k], o);
    if ((threadIdx.x & 31) == 0) sh[k][threadIdx.x >> 5] = sum[k];
  }
  __syncthreads();
  float qs = 0.f, ks = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) { qs += sh[0][w]; ks += sh[1][w]; }
  auto put = [&](const float* src, const T* w, T* dst, int n, int width, float inv) {
    for (int i = threadIdx.x * VEC; i < width; i += blockDim.x * VEC) {
      float v[VEC];
      if (i < n) {                                         // (n is a multiple of VEC)
        ldv<DT, VEC>(w + i, v);
#pragma unroll
        for (int j = 0; j < VEC; ++j) v[j] *= src[i + j] * inv;
      } else {
#pragma unroll
        for (int j = 0; j < VEC; ++j) v[j] = 0.f;
      }
      stv<DT, VEC>(dst + i, v);
    }
  };
  if (p.q_rank > 0)
    put(row, reinterpret_cast<const T*>(p.q_norm), reinterpret_cast<T*>(p.cq) + (size_t)t * p.q_pad, p.q_rank, p.q_pad, 1.0f / sqrtf(qs / (float)p.q_rank + p.eps));
  put(krow, reinterpret_cast<const T*>(p.kv_norm), yp, p.rank, p.lv, 1.0f / sqrtf(ks / (float)p.rank + p.eps));
}

// dst[t, h, :width] = src[t, h, :width] with the first `rot` dimensions turned, pairs (2j, 2j + 1) or (neox) (j, j + rot / 2); dst may be src
struct RopeHeadsParams {
  const void* src; void* dst;
  long long ld_src, ld_dst;
  int T, H, head_src, head_dst, rot, width, neox, tab_rows;
  const int* positions;
  const float* cos_tab; const float* sin_tab;
};

template <int DT>
__global__ void __launch_bounds__(256) rope_heads_kernel(const RopeHeadsParams p) {
  typedef typename Act<DT>::T T;
  pdl_launch_dependents();
  pdl_wait();
  const int pairs = p.width >> 1, half = p.rot >> 1;
  const long long total = (long long)p.T * p.H * pairs;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int j = (int)(i % pairs), h = (int)(i / pairs % p.H), t = (int)(i / pairs / p.H);
    const T* s = reinterpret_cast<const T*>(p.src) + (size_t)t * p.ld_src + (size_t)h * p.head_src;
    T* d = reinterpret_cast<T*>(p.dst) + (size_t)t * p.ld_dst + (size_t)h * p.head_dst;
    const bool halves = p.neox && j < half;
    const int i0 = halves ? j : 2 * j, i1 = halves ? j + half : 2 * j + 1;
    float u = Act<DT>::ld(s[i0]), v = Act<DT>::ld(s[i1]);
    if (j < half) {
      int pos = p.positions[t];
      pos = pos < 0 ? 0 : (pos >= p.tab_rows ? p.tab_rows - 1 : pos);
      const float c = p.cos_tab[(size_t)pos * half + j], sn = p.sin_tab[(size_t)pos * half + j], u0 = u;
      u = u0 * c - v * sn;
      v = v * c + u0 * sn;
    }
    d[i0] = Act<DT>::st(u);
    d[i1] = Act<DT>::st(v);
  }
}

// The end of a layer whose mixer and feed-forward stand side by side, each behind the sigmoid of its own logits, and the norms that open
// the next one:
//   h[t] += sigmoid(g1[t]) * y1[t] + sigmoid(g2[t]) * sum_k wts[t, k] ys[pos[t, k]]       (pos == nullptr: ys[t]; either part may be absent)
//   x1[t] = Norm(h[t]) * w1,  x2[t] = Norm(h[t]) * w2                                      (w2 may be absent)
// Norm is RMS, or (center) layer norm without bias.  table != nullptr: h[t] starts as the embedding of ids[t].
struct JoinParams {
  float* h;
  const void* table; const int* ids; int vocab;
  const void* y1; const void* g1; long long ld_y1, ld_g1;
  const void* ys; const int* pos; const float* wts; const float* g2; long long ld_g2;
  int topk, H, center;
  const void* w1; const void* w2; void* x1; void* x2;
  float eps;
};

__device__ __forceinline__ float sigmoid32(float z) { return 1.0f / (1.0f + expf(-z)); }

template <int DT, int VEC>
__global__ void gated_join_kernel(const JoinParams p) {
  extern __shared__ float row[];
  __shared__ float sh[2][32];
  pdl_launch_dependents();
  pdl_wait();
  typedef typename Act<DT>::T T;
  const int t = blockIdx.x, H = p.H;
  float* hp = p.h + (size_t)t * H;
  const T* emb = nullptr;
  if (p.table != nullptr) {
    int id = p.ids[t];
    id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    emb = reinterpret_cast<const T*>(p.table) + (size_t)id * H;
  }
  const T* y1 = p.y1 != nullptr ? reinterpret_cast<const T*>(p.y1) + (size_t)t * p.ld_y1 : nullptr;
  const T* g1 = reinterpret_cast<const T*>(p.g1) + (size_t)t * p.ld_g1;
  const T* ys = reinterpret_cast<const T*>(p.ys);
  const float* g2 = p.g2 + (size_t)t * p.ld_g2;
  float sum = 0.f;
  for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {
    float v[VEC], u[VEC], z[VEC];
    if (emb != nullptr) ldv<DT, VEC>(emb + i, v); else ldv<2, VEC>(hp + i, v);
    if (y1 != nullptr) {
      ldv<DT, VEC>(y1 + i, u);
      ldv<DT, VEC>(g1 + i, z);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] += sigmoid32(z[j]) * u[j];
    }
    if (ys != nullptr) {
      float acc[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) acc[j] = 0.f;
      if (p.pos == nullptr) {
        ldv<DT, VEC>(ys + (size_t)t * H + i, acc);
      } else {
#pragma unroll 4
        for (int k = 0; k < p.topk; ++k) {
          const int r = p.pos[(size_t)t * p.topk + k];
          if (r < 0) continue;
          const float wk = p.wts[(size_t)t * p.topk + k];
          ldv<DT, VEC>(ys + (size_t)r * H + i, u);
#pragma unroll
          for (int j = 0; j < VEC; ++j) acc[j] += wk * u[j];
        }
      }
      ldv<2, VEC>(g2 + i, z);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] += sigmoid32(z[j]) * acc[j];
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) { row[i + j] = v[j]; sum += v[j]; }
    if (VEC == 4) st4<2>(hp + i, v); else hp[i] = v[0];
  }
  float mean = 0.f, ss = 0.f;
  if (p.center) mean = block_sum32(sum, sh[0]) / (float)H;
  for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {        // the thread's own columns
#pragma unroll
    for (int j = 0; j < VEC; ++j) { const float d = row[i + j] - mean; ss += d * d; }
  }
  ss = block_sum32(ss, sh[1]);
  const float inv = 1.0f / sqrtf(ss / (float)H + p.eps);
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const T* w = reinterpret_cast<const T*>(k == 0 ? p.w1 : p.w2);
    if (w == nullptr) continue;
    T* x = reinterpret_cast<T*>(k == 0 ? p.x1 : p.x2) + (size_t)t * H;
    for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {
      float wv[VEC], o[VEC];
      ldv<DT, VEC>(w + i, wv);
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = (row[i + j] - mean) * inv * wv[j];
      if (VEC == 4) st4<DT>(x + i, o); else x[i] = Act<DT>::st(o[0]);
    }
  }
}

// What opens a pass of looped layers: the residual gets a step vector and, where `table` is given, the token's embedding again.
struct PassStart {
  const void* table; const int* ids; const void* vec; int vocab;
};

// z[t] = sum_k wk * ys[pos[t, k]] + shared[t]; with an output norm z = RMSNorm(z) * post; h[t] += alpha * z (+ pass start); then
// y[t] = RMSNorm(h[t]) * w.  wts == nullptr: every weight is `wconst`.  pos == nullptr: z[t] = ys[t] (ys == nullptr: nothing).
// w == nullptr: y[t] = h[t].  y == nullptr: h only.
template <int DT, int VEC>
__global__ void moe_combine_norm32_kernel(const typename Act<DT>::T* __restrict__ ys, const int* __restrict__ pos, const float* __restrict__ wts,
                                          float wconst, const typename Act<DT>::T* __restrict__ shared_y, float* __restrict__ h,
                                          const typename Act<DT>::T* __restrict__ post, const typename Act<DT>::T* __restrict__ w,
                                          typename Act<DT>::T* __restrict__ y, int topk, int H, float alpha, float eps, const PassStart ps) {
  extern __shared__ float row[];
  __shared__ float sh[2][32];
  pdl_launch_dependents();
  pdl_wait();
  typedef typename Act<DT>::T T;
  const int t = blockIdx.x;
  float* hp = h + (size_t)t * H;
  const T* pvec = reinterpret_cast<const T*>(ps.vec);
  const T* pemb = nullptr;
  if (ps.table != nullptr) {
    int id = ps.ids[t];
    id = id < 0 ? 0 : (id >= ps.vocab ? ps.vocab - 1 : id);
    pemb = reinterpret_cast<const T*>(ps.table) + (size_t)id * H;
  }
  auto start = [&](float* v, int i) {                  // adds the pass start's columns i .. i + VEC - 1
    float u[VEC];
    if (pemb != nullptr) {
      if (VEC == 4) ld4<DT>(pemb + i, u); else u[0] = Act<DT>::ld(pemb[i]);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] += u[j];
    }
    if (pvec != nullptr) {
      if (VEC == 4) ld4<DT>(pvec + i, u); else u[0] = Act<DT>::ld(pvec[i]);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] += u[j];
    }
  };
  float ss = 0.f;
  for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {
    float acc[VEC], v[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) acc[j] = 0.f;
    if (pos == nullptr) {
      if (ys == nullptr) {
      } else if (VEC == 4) ld4<DT>(ys + (size_t)t * H + i, acc); else acc[0] = Act<DT>::ld(ys[(size_t)t * H + i]);
    } else {
      for (int k = 0; k < topk; ++k) {
        const int r = pos[(size_t)t * topk + k];
        if (r < 0) continue;
        const float wk = wts != nullptr ? wts[(size_t)t * topk + k] : wconst;
        if (VEC == 4) ld4<DT>(ys + (size_t)r * H + i, v); else v[0] = Act<DT>::ld(ys[(size_t)r * H + i]);
#pragma unroll
        for (int j = 0; j < VEC; ++j) acc[j] += wk * v[j];
      }
    }
    if (shared_y != nullptr) {
      if (VEC == 4) ld4<DT>(shared_y + (size_t)t * H + i, v); else v[0] = Act<DT>::ld(shared_y[(size_t)t * H + i]);
#pragma unroll
      for (int j = 0; j < VEC; ++j) acc[j] += v[j];
    }
    if (post != nullptr) {                     // the thread's own columns wait in shared memory for the output norm
#pragma unroll
      for (int j = 0; j < VEC; ++j) { ss += acc[j] * acc[j]; row[i + j] = acc[j]; }
      continue;
    }
    if (VEC == 4) ld4<2>(hp + i, v); else v[0] = hp[i];
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] += alpha * acc[j];
    start(v, i);
#pragma unroll
    for (int j = 0; j < VEC; ++j) { ss += v[j] * v[j]; row[i + j] = v[j]; }
    if (VEC == 4) st4<2>(hp + i, v); else hp[i] = v[0];
  }
  if (post != nullptr) {
    ss = block_sum32(ss, sh[0]);
    const float inv = 1.0f / sqrtf(ss / (float)H + eps);
    ss = 0.f;
    for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {
      float pv[VEC], v[VEC];
      if (VEC == 4) { ld4<DT>(post + i, pv); ld4<2>(hp + i, v); } else { pv[0] = Act<DT>::ld(post[i]); v[0] = hp[i]; }
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] += alpha * (row[i + j] * inv * pv[j]);
      start(v, i);
#pragma unroll
      for (int j = 0; j < VEC; ++j) { ss += v[j] * v[j]; row[i + j] = v[j]; }
      if (VEC == 4) st4<2>(hp + i, v); else hp[i] = v[0];
    }
  }
  if (y == nullptr) return;
  float inv = 1.f;
  if (w != nullptr) {
    ss = block_sum32(ss, sh[1]);
    inv = 1.0f / sqrtf(ss / (float)H + eps);
  }
  row_write<DT, VEC>(row, w, y + (size_t)t * H, H, inv);       // (without a weight every thread writes the columns it owns)
}

// xs[pos[t, k]] = wts[t, k] * x[t] for fp32 rows: one CTA per row, all its experts' copies
template <int DT, int VEC>
__global__ void moe_gather_scaled_kernel(const float* __restrict__ x, const int* __restrict__ pos, const float* __restrict__ wts,
                                         typename Act<DT>::T* __restrict__ xs, int topk, int H) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  for (int i = threadIdx.x * VEC; i < H; i += blockDim.x * VEC) {
    float v[VEC], o[VEC];
    if (VEC == 4) ld4<2>(x + (size_t)t * H + i, v); else v[0] = x[(size_t)t * H + i];
    for (int k = 0; k < topk; ++k) {
      const int r = pos[(size_t)t * topk + k];
      if (r < 0) continue;
      const float wk = wts[(size_t)t * topk + k];
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = wk * v[j];
      if (VEC == 4) st4<DT>(xs + (size_t)r * H + i, o); else xs[(size_t)r * H + i] = Act<DT>::st(o[0]);
    }
  }
}

// Per-head RMS norm, rotary positions and cache append of a merged projection [queries | gate | keys | values], one warp per (token,
// head), fp32 arithmetic.  Heads are D wide, stored Dp (values Vp); queries are rewritten in place, keys and values go to their cache
// slots (slot < 0: nowhere).  rot: leading dimensions that turn, in pairs (2j, 2j + 1) or (neox) (j, j + rot / 2); cos / sin tables
// [tab_rows, rot / 2].  Norm weights null: no norm, or (unit) one without weights; with neither norm nor rotation the queries stay as
// they are.  A rotation keeps a head's root mean square, so the norm may stand before or after it.  rot_v: leading dimensions of a
// value that turn, in pairs (2j, 2j + 1), by tables of their own.
struct HeadPostParams {
  void* proj; long long ld;
  const int* positions; const int* slots;
  int T, H, G, D, Dp, Vp, k_col, v_col, rot, neox;
  const void* q_norm; const void* k_norm;
  int unit;
  const float* cos_tab; const float* sin_tab;
  int rot_v;
  const float* cos_v; const float* sin_v;
  int tab_rows, num_slots;
  void* k_pool; void* v_pool;
  float eps;
};

// PAIRS: with norm weights and pairs (2j, 2j + 1), the common form
template <int DT, bool PAIRS>
__global__ void __launch_bounds__(256) head_norm_rope_kernel(const HeadPostParams p) {
  typedef typename Act<DT>::T T;
  pdl_launch_dependents();
  pdl_wait();
  const int h0 = !PAIRS && p.q_norm == nullptr && !p.unit && p.rot == 0 ? p.H : 0;        // first head there is work for
  const int units = p.H + 2 * p.G - h0;
  const long long u = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (u >= (long long)p.T * units) return;
  const int lane = threadIdx.x & 31;
  const int t = (int)(u / units), k = h0 + (int)(u - (long long)t * units);
  T* row = reinterpret_cast<T*>(p.proj) + (size_t)t * p.ld;
  const int slot = p.slots[t];
  const bool cached = slot >= 0 && slot < p.num_slots;
  if (k >= p.H + p.G) {                                    // values
    if (!cached) return;
    const int g = k - p.H - p.G;
    const T* src = row + p.v_col + g * p.Vp;
    T* dst = reinterpret_cast<T*>(p.v_pool) + ((size_t)slot * p.G + g) * p.Vp;
    if (!PAIRS && p.rot_v > 0) {
      int pos = p.positions[t];
      pos = pos < 0 ? 0 : (pos >= p.tab_rows ? p.tab_rows - 1 : pos);
      const int half = p.rot_v >> 1;
      for (int j = lane; 2 * j < p.Vp; j += 32) {
        float a = Act<DT>::ld(src[2 * j]), b = Act<DT>::ld(src[2 * j + 1]);
        if (j < half) {
          const float c = p.cos_v[(size_t)pos * half + j], s = p.sin_v[(size_t)pos * half + j], u0 = a;
          a = u0 * c - b * s;
          b = b * c + u0 * s;
        }
        dst[2 * j] = Act<DT>::st(a);
        dst[2 * j + 1] = Act<DT>::st(b);
      }
      return;
    }
    for (int i = lane; i < p.Vp; i += 32) dst[i] = src[i];
    return;
  }
  const bool is_k = k >= p.H;
  if (is_k && !cached) return;
  T* src = is_k ? row + p.k_col + (k - p.H) * p.Dp : row + (size_t)k * p.Dp;
  T* dst = is_k ? reinterpret_cast<T*>(p.k_pool) + ((size_t)slot * p.G + (k - p.H)) * p.Dp : src;
  const T* nw = reinterpret_cast<const T*>(is_k ? p.k_norm : p.q_norm);
  const bool norm = PAIRS || nw != nullptr || p.unit;
  float inv = 1.f;
  if (norm) {
    float ss = 0.f;
    for (int i = lane; i < p.D; i += 32) { const float v = Act<DT>::ld(src[i]); ss += v * v; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    inv = 1.0f / sqrtf(ss / (float)p.D + p.eps);
  }
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.tab_rows ? p.tab_rows - 1 : pos);
  const int half = p.rot >> 1;
  const float* ct = p.cos_tab + (size_t)pos * half;
  const float* st = p.sin_tab + (size_t)pos * half;
  for (int j = lane; 2 * j < p.Dp; j += 32) {              // pairs (Dp is even; beyond D the row is zero and stays zero)
    const bool halves = !PAIRS && p.neox && j < half;
    const int i0 = halves ? j : 2 * j, i1 = halves ? j + half : 2 * j + 1;
    float a = i0 < p.D ? Act<DT>::ld(src[i0]) * inv : 0.f;
    float b = i1 < p.D ? Act<DT>::ld(src[i1]) * inv : 0.f;
    if (PAIRS || nw != nullptr) {
      if (i0 < p.D) a *= Act<DT>::ld(nw[i0]);
      if (i1 < p.D) b *= Act<DT>::ld(nw[i1]);
    }
    if (j < half) {
      const float c = ct[j], s = st[j], u0 = a;
      a = u0 * c - b * s;
      b = b * c + u0 * s;
    }
    dst[i0] = Act<DT>::st(a);
    dst[i1] = Act<DT>::st(b);
  }
}

// dst[i] = src[idx[i]] for rows of `vecs` 16-byte units
__global__ void gather_rows_kernel(const uint4* __restrict__ src, const long long* __restrict__ idx, uint4* __restrict__ dst, int rows, int vecs) {
  const long long total = (long long)rows * vecs;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int r = (int)(i / vecs), c = (int)(i - (long long)r * vecs);
    dst[i] = src[idx[r] * vecs + c];
  }
}

constexpr int S32_MAX_ROW = 49152;           // floats of the shared-memory row buffer
static int row_threads(int H, int vec) {
  int n = (H / vec + 31) / 32 * 32;
  return n < 64 ? 64 : n > 512 ? 512 : n;
}

}  // namespace fb

using namespace fb;

#define S32_LAUNCH(kern, grid, threads, H, stream, ...)                                                                            \
  {                                                                                                                                \
    static DeviceOnce cfg_;                                                                                                        \
    if (cfg_.need()) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, S32_MAX_ROW * 4);                     \
    launch_k(kern, dim3(grid), dim3(threads), (size_t)(H) * 4, reinterpret_cast<cudaStream_t>(stream), 0, __VA_ARGS__);             \
  }

extern "C" int fb_rmsnorm32(const float* x, const void* w, void* y, int M, int H, int ldx, int ldy, float eps, int dt, void* stream) {
  if (M <= 0) return 0;
  if (H <= 0 || H > S32_MAX_ROW || dt < 0 || dt > 2) return -1;
  const bool vec = H % 4 == 0 && ldx % 4 == 0 && ldy % 4 == 0;
  const int th = row_threads(H, vec ? 4 : 1);
#define GO(DT, V) S32_LAUNCH((rmsnorm32_kernel<DT, V>), M, th, H, stream, x, (const Act<DT>::T*)w, (Act<DT>::T*)y, H, ldx, ldy, eps)
  if (vec) { if (dt == 0) GO(0, 4) else if (dt == 1) GO(1, 4) else GO(2, 4) }
  else { if (dt == 0) GO(0, 1) else if (dt == 1) GO(1, 1) else GO(2, 1) }
#undef GO
  return (int)cudaGetLastError();
}

extern "C" int fb_embed_pos_norm(const int* ids, const int* positions, const void* table, const double* inv_freq, const void* pos_table,
                                 int pos_rows, const void* add_vec, const void* w, float* h, void* y, int T, int H, int vocab, float eps, int dt, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || H > S32_MAX_ROW || dt < 0 || dt > 2 || (pos_table != nullptr && pos_rows <= 0)) return -1;
  const bool vec = H % 4 == 0;
  const int th = row_threads(H, vec ? 4 : 2);
#define GO(DT, V) S32_LAUNCH((embed_pos_norm_kernel<DT, V>), T, th, H, stream, ids, positions, (const Act<DT>::T*)table, inv_freq, (const Act<DT>::T*)pos_table, pos_rows, (const Act<DT>::T*)add_vec, (const Act<DT>::T*)w, h, (Act<DT>::T*)y, H, vocab, eps)
  if (vec) { if (dt == 0) GO(0, 4) else if (dt == 1) GO(1, 4) else GO(2, 4) }
  else { if (dt == 0) GO(0, 1) else if (dt == 1) GO(1, 1) else GO(2, 1) }
#undef GO
  return (int)cudaGetLastError();
}

// See LatentPostParams.
extern "C" int fb_latent_post(const void* x, long long ldx, int q_col, int q_rank, int q_pad, int kv_col, int rank, int lv, int rot_col, int rot, int ld, int neox,
                              int gate_col, int n_gates, const void* q_norm, const void* kv_norm, const float* cos_tab, const float* sin_tab, int tab_rows,
                              const int* positions, const int* slots, void* cq, void* pool, float* gates, int T, long long spare, float eps, int dt,
                              void* stream) {
  if (T <= 0) return 0;
  if (rank <= 0 || lv < rank || ld < lv + rot || q_rank < 0 || q_pad < q_rank || q_rank + rank > S32_MAX_ROW || rot < 0 || (rot & 1) || ((ld - lv) & 1) || n_gates < 0 ||
      dt < 0 || dt > 2 || (rot == 0 && ld != lv) || (rot > 0 && (cos_tab == nullptr || sin_tab == nullptr || positions == nullptr || tab_rows <= 0)) ||
      (q_rank > 0 && (cq == nullptr || q_norm == nullptr)) || (n_gates > 0 && gates == nullptr))
    return -1;
  LatentPostParams p{x, ldx, q_col, q_rank, q_pad, kv_col, rank, lv, rot_col, rot, ld, neox, gate_col, n_gates, q_norm, kv_norm, cos_tab, sin_tab, tab_rows, positions, slots, cq, pool, gates, spare, eps};
  const bool vec = !((q_col | q_rank | q_pad | kv_col | rank | lv | ld | ldx) & 3) && !((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(pool) | reinterpret_cast<uintptr_t>(cq) |
                                                                                         reinterpret_cast<uintptr_t>(q_norm) | reinterpret_cast<uintptr_t>(kv_norm)) & 15);
  const int th = row_threads(ld > q_pad ? ld : q_pad, vec ? 4 : 2);
#define GO(DT, V) S32_LAUNCH((latent_post_kernel<DT, V>), T, th, q_rank + rank, stream, p)
  if (vec) { if (dt == 0) GO(0, 4) else if (dt == 1) GO(1, 4) else GO(2, 4) }
  else { if (dt == 0) GO(0, 1) else if (dt == 1) GO(1, 1) else GO(2, 1) }
#undef GO
  return (int)cudaGetLastError();
}

// See RopeHeadsParams.
extern "C" int fb_rope_heads(const void* src, void* dst, long long ld_src, long long ld_dst, int T, int H, int head_src, int head_dst, int rot, int width, int neox,
                             const int* positions, const float* cos_tab, const float* sin_tab, int tab_rows, int dt, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || rot <= 0 || (rot & 1) || width < rot || (width & 1) || tab_rows <= 0 || cos_tab == nullptr || sin_tab == nullptr || positions == nullptr || dt < 0 || dt > 2) return -1;
  RopeHeadsParams p{src, dst, ld_src, ld_dst, T, H, head_src, head_dst, rot, width, neox, tab_rows, positions, cos_tab, sin_tab};
  long long blocks = ((long long)T * H * (width / 2) + 255) / 256;
  if (blocks > 148 * 32) blocks = 148 * 32;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (dt == 0) launch_k(rope_heads_kernel<0>, dim3((unsigned)blocks), dim3(256), 0, s, 0, p);
  else if (dt == 1) launch_k(rope_heads_kernel<1>, dim3((unsigned)blocks), dim3(256), 0, s, 0, p);
  else launch_k(rope_heads_kernel<2>, dim3((unsigned)blocks), dim3(256), 0, s, 0, p);
  return (int)cudaGetLastError();
}

// See JoinParams; x1 / x2 [T, H] and ys rows are contiguous.
extern "C" int fb_gated_join(float* h, const void* table, const int* ids, int vocab, const void* y1, long long ld_y1, const void* g1, long long ld_g1, const void* ys,
                             const int* pos, const float* wts, const float* g2, long long ld_g2, int T, int topk, int H, int center, const void* w1,
                             const void* w2, void* x1, void* x2, float eps, int dt, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || H > S32_MAX_ROW || dt < 0 || dt > 2 || w1 == nullptr || x1 == nullptr || (w2 != nullptr && x2 == nullptr) || (y1 != nullptr && g1 == nullptr) ||
      (ys != nullptr && g2 == nullptr) || (pos != nullptr && (wts == nullptr || topk <= 0)) || (table != nullptr && (ids == nullptr || vocab <= 0)))
    return -1;
  JoinParams p{h, table, ids, vocab, y1, g1, ld_y1, ld_g1, ys, pos, wts, g2, ld_g2, topk, H, center, w1, w2, x1, x2, eps};
  const uintptr_t align = dt == 2 ? 15 : 7;
  const bool vec = H % 4 == 0 && ld_y1 % 4 == 0 && ld_g1 % 4 == 0 && ld_g2 % 4 == 0 && !(reinterpret_cast<uintptr_t>(g2) & 15) &&
                   !((reinterpret_cast<uintptr_t>(y1) | reinterpret_cast<uintptr_t>(g1) | reinterpret_cast<uintptr_t>(ys)) & align);
  const int th = row_threads(H, vec ? 4 : 1);
#define GO(DT, V) S32_LAUNCH((gated_join_kernel<DT, V>), T, th, H, stream, p)
  if (vec) { if (dt == 0) GO(0, 4) else if (dt == 1) GO(1, 4) else GO(2, 4) }
  else { if (dt == 0) GO(0, 1) else if (dt == 1) GO(1, 1) else GO(2, 1) }
#undef GO
  return (int)cudaGetLastError();
}

extern "C" int fb_moe_combine_norm32(const void* ys, const int* pos, const float* wts, float wconst, const void* shared_y, float* h,
                                     const void* post, const void* w, void* y, int T, int topk, int H, float alpha, float eps,
                                     const void* start_table, const int* ids, int vocab, const void* start_vec, int dt, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || H > S32_MAX_ROW || dt < 0 || dt > 2 || (pos != nullptr && ys == nullptr) || (start_table != nullptr && (ids == nullptr || vocab <= 0))) return -1;
  const PassStart ps{start_table, ids, start_vec, vocab};
  const bool vec = H % 4 == 0;
  const int th = row_threads(H, vec ? 4 : 1);
#define GO(DT, V) S32_LAUNCH((moe_combine_norm32_kernel<DT, V>), T, th, H, stream, (const Act<DT>::T*)ys, pos, wts, wconst, (const Act<DT>::T*)shared_y, h, (const Act<DT>::T*)post, (const Act<DT>::T*)w, (Act<DT>::T*)y, topk, H, alpha, eps, ps)
  if (vec) { if (dt == 0) GO(0, 4) else if (dt == 1) GO(1, 4) else GO(2, 4) }
  else { if (dt == 0) GO(0, 1) else if (dt == 1) GO(1, 1) else GO(2, 1) }
#undef GO
  return (int)cudaGetLastError();
}

extern "C" int fb_gather_rows(const void* src, const long long* idx, void* dst, int rows, int row_bytes, void* stream) {
  if (rows <= 0) return 0;
  if (row_bytes <= 0 || row_bytes % 16 != 0) return -1;
  const int vecs = row_bytes / 16;
  long long blocks = ((long long)rows * vecs + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  launch_k(gather_rows_kernel, dim3((unsigned)blocks), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), 0, (const uint4*)src, idx, (uint4*)dst, rows, vecs);
  return (int)cudaGetLastError();
}

// x: fp32 [T, H]; xs: sorted rows of type dt.
extern "C" int fb_moe_gather_scaled(const float* x, const int* pos, const float* wts, void* xs, int T, int topk, int H, int dt, void* stream_) {
  if (T <= 0) return 0;
  if (H <= 0 || topk <= 0 || dt < 0 || dt > 2) return -1;
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  const bool vec = H % 4 == 0;
  const int th = row_threads(H, vec ? 4 : 1);
#define GO(DT, V) launch_k(moe_gather_scaled_kernel<DT, V>, dim3(T), dim3(th), 0, stream, 0, x, pos, wts, (Act<DT>::T*)xs, topk, H)
  if (vec) { if (dt == 0) GO(0, 4); else if (dt == 1) GO(1, 4); else GO(2, 4); }
  else { if (dt == 0) GO(0, 1); else if (dt == 1) GO(1, 1); else GO(2, 1); }
#undef GO
  return (int)cudaGetLastError();
}

// See HeadPostParams.  G = 0: queries only (the layer reads another layer's cache).
extern "C" int fb_head_norm_rope(void* proj, long long ld, const int* positions, const int* slots, int T, int H, int G, int D, int Dp, int Vp,
                                 int k_col, int v_col, int rot, int neox, const void* q_norm, const void* k_norm, int unit, const float* cos_tab,
                                 const float* sin_tab, int rot_v, const float* cos_v, const float* sin_v, int tab_rows, int num_slots, void* k_pool, void* v_pool, float eps, int dt, void* stream_) {
  if (T <= 0) return 0;
  if (H <= 0 || G < 0 || D <= 0 || Dp < D || (Dp & 1) || Vp <= 0 || rot < 0 || (rot & 1) || rot > D || dt < 0 || dt > 2) return -1;
  if (rot > 0 && (cos_tab == nullptr || sin_tab == nullptr || tab_rows <= 0)) return -1;
  if (rot_v < 0 || (rot_v & 1) || rot_v > Vp || (rot_v > 0 && (cos_v == nullptr || sin_v == nullptr || tab_rows <= 0 || (Vp & 1)))) return -1;
  if (unit && q_norm != nullptr) return -1;
  if (G > 0 && ((k_norm == nullptr) != (q_norm == nullptr) || k_pool == nullptr || v_pool == nullptr)) return -1;
  HeadPostParams p{proj, ld, positions, slots, T, H, G, D, Dp, Vp, k_col, v_col, rot, neox, q_norm, k_norm, unit, cos_tab, sin_tab, rot_v, cos_v, sin_v, tab_rows, num_slots, k_pool, v_pool, eps};
  const long long units = (long long)T * ((q_norm == nullptr && !unit && rot == 0 ? 0 : H) + 2 * G);
  if (units == 0) return 0;
  const dim3 grid((unsigned)((units + 7) / 8));
  cudaStream_t stream = reinterpret_cast<cudaStream_t>(stream_);
  const bool pairs = q_norm != nullptr && !neox && rot_v == 0;
#define GO(DT) { if (pairs) launch_k(head_norm_rope_kernel<DT, true>, grid, dim3(256), 0, stream, 0, p); else launch_k(head_norm_rope_kernel<DT, false>, grid, dim3(256), 0, stream, 0, p); }
  if (dt == 0) GO(0) else if (dt == 1) GO(1) else GO(2)
#undef GO
  return (int)cudaGetLastError();
}
