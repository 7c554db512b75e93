// Shared pieces of the kernels that work on hybrid (recurrent + attention) layers: element-type helpers, the accessor
// for a projection that is either a finished matrix or the fp32 slabs of a split-K GEMM, and the step descriptor.
#pragma once
#include "ptx.cuh"

namespace b200 {

__device__ __forceinline__ float to_f(float x) { return x; }
__device__ __forceinline__ float to_f(__nv_bfloat16 x) { return __bfloat162float(x); }
template <typename T>
__device__ __forceinline__ T from_f(float x);
template <>
__device__ __forceinline__ float from_f<float>(float x) { return x; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float x) { return __float2bfloat16_rn(x); }
template <typename T>
__device__ __forceinline__ float round_to(float x) { return to_f(from_f<T>(x)); }

// Four consecutive elements as fp32 (the address is 4-element aligned).
__device__ __forceinline__ void load4(const float* p, float* f) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float* f) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
}
__device__ __forceinline__ void store4(float* p, const float* f) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float* f) {
  uint2 u;
  u.x = pack_bf16x2(f[0], f[1]);
  u.y = pack_bf16x2(f[2], f[3]);
  *reinterpret_cast<uint2*>(p) = u;
}

// A projection's output [rows, ld]: a matrix of the activation type, or (ws != null) `splits` fp32 slabs that are
// summed on the way in and rounded to the activation type. Every consumer of a fused input projection takes one.
template <typename T>
struct Proj {
  const T* p;
  const float* ws;
  int splits;
  long long slab;
  int ld;
  __device__ __forceinline__ float get(int row, int col) const {
    const size_t i = (size_t)row * ld + col;
    if (ws == nullptr) return to_f(p[i]);
    float v = ws[i];
    for (int s = 1; s < splits; ++s) v += ws[(size_t)s * slab + i];
    return round_to<T>(v);
  }
  // the same without the rounding, for values that enter 32-bit arithmetic directly (step sizes)
  __device__ __forceinline__ float get_raw(int row, int col) const {
    const size_t i = (size_t)row * ld + col;
    if (ws == nullptr) return to_f(p[i]);
    float v = ws[i];
    for (int s = 1; s < splits; ++s) v += ws[(size_t)s * slab + i];
    return v;
  }
  __device__ __forceinline__ void get4(int row, int col, float* f) const {   // col and ld multiples of 4
    const size_t i = (size_t)row * ld + col;
    if (ws == nullptr) { load4(p + i, f); return; }
    load4(ws + i, f);
    for (int s = 1; s < splits; ++s) {
      float g[4];
      load4(ws + (size_t)s * slab + i, g);
#pragma unroll
      for (int k = 0; k < 4; ++k) f[k] += g[k];
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) f[k] = round_to<T>(f[k]);
  }
};

template <typename T>
inline Proj<T> make_proj(const void* p, const float* ws, int splits, long long slab, int ld) {
  Proj<T> r;
  r.p = reinterpret_cast<const T*>(p);
  r.ws = ws;
  r.splits = splits;
  r.slab = slab;
  r.ld = ld;
  return r;
}

// The ragged batch of one model step: `n` sequences, sequence i brings the tokens [cu[i], cu[i+1]) of the packed stream,
// they sit at positions start[i].. of its context, and its recurrent state lives in row seq_row[i] of the state pools.
// active (optional): sequences with a zero entry leave every state untouched.
struct Ragged {
  const int* cu;
  const int* start;
  const int* row;
  const int* active;
  const int* tok_seq;   // [T] sequence of every token
  int n, T;
  __device__ __forceinline__ bool live(int i) const { return active == nullptr || active[i] != 0; }
};
inline Ragged make_ragged(const int* cu, const int* start, const int* row, const int* active, const int* tok_seq, int n,
                          int T) {
  Ragged r;
  r.cu = cu; r.start = start; r.row = row; r.active = active; r.tok_seq = tok_seq; r.n = n; r.T = T;
  return r;
}

__device__ __forceinline__ float silu_f(float v) { return __fdividef(v, 1.f + __expf(-v)); }
// log(1 + e^x) without overflow; both branches keep the relative accuracy of small results.
__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

template <int THREADS>
__device__ __forceinline__ float block_sum_all(float v, float* red /*[32]*/) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = l < THREADS / 32 ? red[l] : 0.f;
  t = warp_sum(t);
  __syncthreads();
  return t;
}

}  // namespace b200
