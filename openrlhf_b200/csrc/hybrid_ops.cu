// Elementwise and row-wise steps of hybrid decoder layers whose residual stream is fp32 and whose sublayers read one
// shared norm: embedding to fp32, RMS norm of an fp32 row, squared-ReLU, logit soft-capping, rotary embedding (on a
// leading part of each head) with KV-cache write, gated group RMS norm, and the fused tails of split-K projections
// (reduce + residual + norm). T is the activation type: bf16 when serving, float for the all-32-bit mode.
#include "proj.cuh"

namespace b200 {

constexpr int HY_THREADS = 256;

// ------------------------------------------------------------------ embedding
template <typename T>
__global__ void embed_f32_kernel(const long long* __restrict__ ids, const T* __restrict__ table, float* __restrict__ x,
                                 int n_tok, int ld, int vocab) {
  const int nv = ld >> 2;
  const long long total = (long long)n_tok * nv;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / nv), v = (int)(i % nv);
    long long id = ids[t];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    float f[4];
    load4(table + (size_t)id * ld + 4 * v, f);
    store4(x + (size_t)t * ld + 4 * v, f);
  }
}

// ------------------------------------------------------------------ RMS norm of fp32 rows (optionally gathered)
// x [*, ld] fp32, n real columns (the padding of x is zero); y [M, ld]: x * rsqrt(mean(x^2) + eps) * w.
// With slabs: x += sum over the split-K slabs first (residual add), written back.
template <typename T>
__global__ void __launch_bounds__(HY_THREADS)
rmsnorm_f32_kernel(float* __restrict__ x, const float* __restrict__ ws, int splits, long long slab,
                   const int* __restrict__ rows, const T* __restrict__ w, T* __restrict__ y, int M, int n, int ld,
                   float eps) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float row_buf[];
  __shared__ float red[32];
  const int nv = ld >> 2;
  for (int m = blockIdx.x; m < M; m += gridDim.x) {
    const size_t src = (size_t)(rows != nullptr ? rows[m] : m) * ld;
    float ss = 0.f;
    for (int v = threadIdx.x; v < nv; v += HY_THREADS) {
      float f[4];
      load4(x + src + 4 * v, f);
      if (ws != nullptr) {
        for (int s = 0; s < splits; ++s) {
          float g[4];
          load4(ws + (size_t)s * slab + src + 4 * v, g);
#pragma unroll
          for (int k = 0; k < 4; ++k) f[k] += g[k];
        }
        store4(x + src + 4 * v, f);
      }
      store4(row_buf + 4 * v, f);
#pragma unroll
      for (int k = 0; k < 4; ++k) ss += f[k] * f[k];
    }
    ss = block_sum_all<HY_THREADS>(ss, red);
    const float rstd = 1.f / sqrtf(ss / (float)n + eps);
    for (int v = threadIdx.x; v < nv; v += HY_THREADS) {
      float f[4], g[4];
      load4(row_buf + 4 * v, f);
      load4(w + 4 * v, g);
#pragma unroll
      for (int k = 0; k < 4; ++k) f[k] = f[k] * rstd * g[k];
      store4(y + (size_t)m * ld + 4 * v, f);
    }
    __syncthreads();
  }
}

// Long batches without slabs: one warp per row, the row in registers (ld up to 32 * 4 * NV).
template <typename T, int NV>
__global__ void __launch_bounds__(HY_THREADS)
rmsnorm_f32_warp_kernel(const float* __restrict__ x, const T* __restrict__ w, T* __restrict__ y, int M, int n, int ld,
                        float eps) {
  const int lane = threadIdx.x & 31;
  for (int m = blockIdx.x * (HY_THREADS / 32) + (threadIdx.x >> 5); m < M; m += gridDim.x * (HY_THREADS / 32)) {
    float f[NV][4];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * 32 + lane) * 4;
      if (c < ld) load4(x + (size_t)m * ld + c, f[i]);
      else f[i][0] = f[i][1] = f[i][2] = f[i][3] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int k = 0; k < 4; ++k) ss += f[i][k] * f[i][k];
    const float rstd = 1.f / sqrtf(warp_sum(ss) / (float)n + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * 32 + lane) * 4;
      if (c < ld) {
        float g[4];
        load4(w + c, g);
#pragma unroll
        for (int k = 0; k < 4; ++k) f[i][k] = f[i][k] * rstd * g[k];
        store4(y + (size_t)m * ld + c, f[i]);
      }
    }
  }
}

// ------------------------------------------------------------------ logits <- cap * tanh(logits / cap)
__global__ void softcap_kernel(float* __restrict__ x, long long n4, float cap, float inv_cap) {
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n4; i += (long long)gridDim.x * blockDim.x) {
    float f[4];
    load4(x + 4 * i, f);
#pragma unroll
    for (int k = 0; k < 4; ++k) f[k] = cap * tanhf(f[k] * inv_cap);
    store4(x + 4 * i, f);
  }
}

// ------------------------------------------------------------------ rotary embedding + KV write (+ squared ReLU)
// Projection columns [q heads | k heads | v heads]; k / v are absent (kv_heads = 0) when the layer reads another
// layer's cache. Channels [0, rot) of a head rotate in pairs (i, i + rot/2) with the (cos, sin) row of the token's
// position; the rest pass. q -> q_out [T, H, dk_ld]; k, v -> cache slot. Cache and q rows are padded to dk_ld / dv_ld
// (their padding stays zero). One thread per element pair; ff columns are squared-ReLU'd into `ff_dst`.
// The same, four channels at a time (rot / 2, dk - rot and dv multiples of 4) for NT consecutive tokens per thread; all
// loads of a thread are issued before its first store.
template <typename T, int NT>
__global__ void __launch_bounds__(HY_THREADS, 4)
rope_write4_kernel(const Proj<T> src, const int* __restrict__ pos, const int* __restrict__ slots,
                   const float2* __restrict__ table, int max_pos, T* __restrict__ q_out, T* __restrict__ k_cache,
                   T* __restrict__ v_cache, int n_tok, int H, int G, int dk, int dv, int dk_ld, int dv_ld, int rot,
                   int ff_col, int ff, T* __restrict__ ff_dst, int ff_ld) {
  pdl_launch_dependents();
  pdl_wait();
  const int half = rot >> 1;
  const int per_qk = (half + (dk - rot)) >> 2;
  const int n_qk = (H + G) * per_qk, n_v = (G * dv) >> 2, n_f = ff >> 2;
  int e = blockIdx.y * HY_THREADS + threadIdx.x;
  if (e >= n_qk + n_v + n_f) return;
  const int t0 = blockIdx.x * NT;
  float u[NT][4];
  if (e < n_qk) {
    const int head = e / per_qk, i = (e - head * per_qk) * 4, c0 = head * dk;
    const bool turns = i < half;
    float v[NT][4], cs[NT][8];
    int slot[NT];
#pragma unroll
    for (int k = 0; k < NT; ++k) {
      const int t = min(t0 + k, n_tok - 1);
      src.get4(t, c0 + i + (turns ? 0 : half), u[k]);
      if (head >= H) slot[k] = slots[t];
      if (turns) {
        src.get4(t, c0 + i + half, v[k]);
        int p = pos[t];
        p = p < 0 ? 0 : (p >= max_pos ? max_pos - 1 : p);
        const float* row = reinterpret_cast<const float*>(table + (size_t)p * half + i);
        load4(row, cs[k]);
        load4(row + 4, cs[k] + 4);
      }
    }
#pragma unroll
    for (int k = 0; k < NT; ++k) {
      if (t0 + k >= n_tok) break;
      T* dst = head < H ? q_out + ((size_t)(t0 + k) * H + head) * dk_ld : k_cache + ((size_t)slot[k] * G + (head - H)) * dk_ld;
      if (turns) {
        float a[4], b[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          a[j] = u[k][j] * cs[k][2 * j] - v[k][j] * cs[k][2 * j + 1];
          b[j] = v[k][j] * cs[k][2 * j] + u[k][j] * cs[k][2 * j + 1];
        }
        store4(dst + i, a);
        store4(dst + i + half, b);
      } else {
        store4(dst + i + half, u[k]);
      }
    }
  } else if (e < n_qk + n_v) {
    e = (e - n_qk) * 4;
    const int g = e / dv;
    int slot[NT];
#pragma unroll
    for (int k = 0; k < NT; ++k) {
      const int t = min(t0 + k, n_tok - 1);
      src.get4(t, (H + G) * dk + e, u[k]);
      slot[k] = slots[t];
    }
#pragma unroll
    for (int k = 0; k < NT; ++k)
      if (t0 + k < n_tok) store4(v_cache + ((size_t)slot[k] * G + g) * dv_ld + (e - g * dv), u[k]);
  } else {
    e = (e - n_qk - n_v) * 4;
#pragma unroll
    for (int k = 0; k < NT; ++k) src.get4(min(t0 + k, n_tok - 1), ff_col + e, u[k]);
#pragma unroll
    for (int k = 0; k < NT; ++k) {
      if (t0 + k >= n_tok) break;
#pragma unroll
      for (int j = 0; j < 4; ++j) { const float r = fmaxf(u[k][j], 0.f); u[k][j] = r * r; }
      store4(ff_dst + (size_t)(t0 + k) * ff_ld + e, u[k]);
    }
  }
}

template <typename T>
__global__ void rope_write_kernel(const Proj<T> src, const int* __restrict__ pos, const int* __restrict__ slots,
                                  const float2* __restrict__ table, int max_pos, T* __restrict__ q_out,
                                  T* __restrict__ k_cache, T* __restrict__ v_cache, int n_tok, int H, int G, int dk,
                                  int dv, int dk_ld, int dv_ld, int rot, int ff_col, int ff, T* __restrict__ ff_dst,
                                  int ff_ld) {
  pdl_launch_dependents();
  pdl_wait();
  const int half = rot >> 1;
  const int per_qk = half + (dk - rot);             // rotated pairs plus passed channels of one head
  const int n_qk = (H + G) * per_qk, n_v = G * dv, n_f = ff >> 2;
  const int per_tok = n_qk + n_v + n_f;
  const long long total = (long long)n_tok * per_tok;
  for (long long idx = blockIdx.x * (long long)blockDim.x + threadIdx.x; idx < total;
       idx += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(idx / per_tok);
    int e = (int)(idx % per_tok);
    if (e < n_qk) {
      const int head = e / per_qk, i = e % per_qk;
      T* dst;
      if (head < H) dst = q_out + ((size_t)t * H + head) * dk_ld;
      else dst = k_cache + ((size_t)slots[t] * G + (head - H)) * dk_ld;
      const int c0 = head * dk;
      if (i < half) {
        const float u = src.get(t, c0 + i), v = src.get(t, c0 + i + half);
        int p = pos[t];
        p = p < 0 ? 0 : (p >= max_pos ? max_pos - 1 : p);
        const float2 cs = table[(size_t)p * half + i];
        dst[i] = from_f<T>(u * cs.x - v * cs.y);
        dst[i + half] = from_f<T>(v * cs.x + u * cs.y);
      } else {
        dst[i + half] = from_f<T>(src.get(t, c0 + i + half));
      }
    } else if (e < n_qk + n_v) {
      e -= n_qk;
      v_cache[((size_t)slots[t] * G + e / dv) * dv_ld + e % dv] = from_f<T>(src.get(t, (H + G) * dk + e));
    } else {
      e = (e - n_qk - n_v) * 4;
      float f[4];
      src.get4(t, ff_col + e, f);
#pragma unroll
      for (int k = 0; k < 4; ++k) { const float r = fmaxf(f[k], 0.f); f[k] = r * r; }
      store4(ff_dst + (size_t)t * ff_ld + e, f);
    }
  }
}

// ------------------------------------------------------------------ gated group RMS norm (+ squared ReLU)
// dst[t, c] = (y silu(z)) / rms of its group * w; one block per (token, group), an extra block per token takes the
// feed-forward columns. gsize = inner / groups.
template <typename T>
__global__ void __launch_bounds__(HY_THREADS)
gate_norm_kernel(const T* __restrict__ y, const Proj<T> z, const T* __restrict__ w, T* __restrict__ dst, int dst_ld,
                 int n_tok, int inner, int groups, float eps, int ff_col, int ff, T* __restrict__ ff_dst) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float row_buf[];
  __shared__ float red[32];
  const int gsize = inner / groups;
  const int g = blockIdx.y;
  const bool vec = (gsize & 3) == 0 && (inner & 3) == 0 && (z.ld & 3) == 0;
  for (int t = blockIdx.x; t < n_tok; t += gridDim.x) {
    if (g >= groups) {
      for (int c = threadIdx.x * 4; c < ff; c += HY_THREADS * 4) {
        float f[4];
        z.get4(t, ff_col + c, f);
#pragma unroll
        for (int k = 0; k < 4; ++k) { const float r = fmaxf(f[k], 0.f); f[k] = r * r; }
        store4(ff_dst + (size_t)t * dst_ld + c, f);
      }
      continue;
    }
    const int c0 = g * gsize;
    float ss = 0.f;
    if (vec) {
      for (int c = threadIdx.x * 4; c < gsize; c += HY_THREADS * 4) {
        float f[4], zz[4];
        load4(y + (size_t)t * inner + c0 + c, f);
        z.get4(t, c0 + c, zz);
#pragma unroll
        for (int k = 0; k < 4; ++k) { f[k] *= silu_f(zz[k]); ss += f[k] * f[k]; }
        store4(row_buf + c, f);
      }
    } else {
      for (int c = threadIdx.x; c < gsize; c += HY_THREADS) {
        const float v = to_f(y[(size_t)t * inner + c0 + c]) * silu_f(z.get(t, c0 + c));
        row_buf[c] = v;
        ss += v * v;
      }
    }
    ss = block_sum_all<HY_THREADS>(ss, red);
    const float rstd = 1.f / sqrtf(ss / (float)gsize + eps);
    if (vec) {
      for (int c = threadIdx.x * 4; c < gsize; c += HY_THREADS * 4) {
        float f[4], ww[4];
        load4(row_buf + c, f);
        load4(w + c0 + c, ww);
#pragma unroll
        for (int k = 0; k < 4; ++k) f[k] = f[k] * rstd * ww[k];
        store4(dst + (size_t)t * dst_ld + c0 + c, f);
      }
    } else {
      for (int c = threadIdx.x; c < gsize; c += HY_THREADS)
        dst[(size_t)t * dst_ld + c0 + c] = from_f<T>(row_buf[c] * rstd * to_f(w[c0 + c]));
    }
    __syncthreads();
  }
}

static inline int hy_grid(long long work, int cap) {
  long long b = (work + HY_THREADS - 1) / HY_THREADS;
  return (int)(b < 1 ? 1 : (b > cap ? cap : b));
}

}  // namespace b200

using namespace b200;
#define HY_STREAM(s) reinterpret_cast<cudaStream_t>(s)
#define HY_OK() (cudaGetLastError() == cudaSuccess ? 0 : -3)

// Every entry point takes `f32`: 1 = activations and weights are float, 0 = bf16.
extern "C" int b200_embed_f32(const long long* ids, const void* table, float* x, int n_tok, int ld, int vocab, int f32,
                              void* stream) {
  if (n_tok <= 0) return 0;
  if (ld % 4) return -10;
  const int grid = hy_grid((long long)n_tok * (ld / 4), 148 * 16);
  if (f32) embed_f32_kernel<float><<<grid, HY_THREADS, 0, HY_STREAM(stream)>>>(ids, (const float*)table, x, n_tok, ld, vocab);
  else embed_f32_kernel<__nv_bfloat16><<<grid, HY_THREADS, 0, HY_STREAM(stream)>>>(ids, (const __nv_bfloat16*)table, x, n_tok, ld, vocab);
  return HY_OK();
}

extern "C" int b200_rmsnorm_f32(float* x, const float* ws, int splits, long long slab, const int* rows, const void* w,
                                void* y, int M, int n, int ld, float eps, int f32, void* stream) {
  if (M <= 0) return 0;
  if (ld % 4 || ld > 12288 || slab % 4 || (ws != nullptr && rows != nullptr)) return -10;
  const int grid = M < 148 * 8 ? M : 148 * 8;
  const size_t smem = (size_t)ld * sizeof(float);
  cudaError_t e;
  if (!f32 && ws == nullptr && rows == nullptr && M >= 1024 && ld <= 4096) {
    typedef __nv_bfloat16 B16;
    const int blocks = (M + 7) / 8 < 148 * 8 ? (M + 7) / 8 : 148 * 8;
    if (ld <= 2048) rmsnorm_f32_warp_kernel<B16, 16><<<blocks, HY_THREADS, 0, HY_STREAM(stream)>>>(x, (const B16*)w, (B16*)y, M, n, ld, eps);
    else rmsnorm_f32_warp_kernel<B16, 32><<<blocks, HY_THREADS, 0, HY_STREAM(stream)>>>(x, (const B16*)w, (B16*)y, M, n, ld, eps);
    return HY_OK();
  }
  if (f32) e = launch_pdl(rmsnorm_f32_kernel<float>, dim3(grid), dim3(HY_THREADS), smem, HY_STREAM(stream), x, ws, splits,
                          slab, rows, (const float*)w, (float*)y, M, n, ld, eps);
  else e = launch_pdl(rmsnorm_f32_kernel<__nv_bfloat16>, dim3(grid), dim3(HY_THREADS), smem, HY_STREAM(stream), x, ws,
                      splits, slab, rows, (const __nv_bfloat16*)w, (__nv_bfloat16*)y, M, n, ld, eps);
  return e == cudaSuccess ? 0 : -3;
}

extern "C" int b200_softcap(float* x, long long n, float cap, void* stream) {
  if (n <= 0) return 0;
  if (n % 4 || !(cap > 0.f)) return -10;
  softcap_kernel<<<hy_grid(n / 4, 148 * 16), HY_THREADS, 0, HY_STREAM(stream)>>>(x, n / 4, cap, 1.f / cap);
  return HY_OK();
}

extern "C" int b200_rope_write(const void* p, const float* ws, int splits, long long slab, int ld, const int* pos,
                               const int* slots, const void* table, int max_pos, void* q_out, void* k_cache,
                               void* v_cache, int n_tok, int H, int G, int dk, int dv, int dk_ld, int dv_ld, int rot,
                               int ff_col, int ff, void* ff_dst, int ff_ld, int f32, void* stream) {
  if (n_tok <= 0) return 0;
  if (rot % 2 || rot > dk || dk_ld < dk || dv_ld < dv || ff % 4 || ff_col % 4 || ld % 4 || ff_ld % 4 || slab % 4) return -10;
  const long long work = (long long)n_tok * ((H + G) * (rot / 2 + dk - rot) + G * dv + ff / 4);
  const bool vec = rot % 8 == 0 && (dk - rot) % 4 == 0 && dv % 4 == 0;
  const int grid = hy_grid(work, 148 * 16);
  const int nt = n_tok >= 512 ? 2 : 1;
  const dim3 grid4((n_tok + nt - 1) / nt, (unsigned)(work / n_tok / (4 * HY_THREADS) + 1));
  cudaError_t e;
#define ROPE_ARGS(TT)                                                                                                 \
  make_proj<TT>(p, ws, splits, slab, ld), pos, slots, (const float2*)table, max_pos, (TT*)q_out, (TT*)k_cache,        \
      (TT*)v_cache, n_tok, H, G, dk, dv, dk_ld, dv_ld, rot, ff_col, ff, (TT*)ff_dst, ff_ld
  if (vec) {
#define ROPE4(TT, NT) \
  launch_pdl(rope_write4_kernel<TT, NT>, grid4, dim3(HY_THREADS), (size_t)0, HY_STREAM(stream), ROPE_ARGS(TT))
    if (f32) e = nt == 2 ? ROPE4(float, 2) : ROPE4(float, 1);
    else e = nt == 2 ? ROPE4(__nv_bfloat16, 2) : ROPE4(__nv_bfloat16, 1);
#undef ROPE4
  } else if (f32) e = launch_pdl(rope_write_kernel<float>, dim3(grid), dim3(HY_THREADS), (size_t)0, HY_STREAM(stream), ROPE_ARGS(float));
  else e = launch_pdl(rope_write_kernel<__nv_bfloat16>, dim3(grid), dim3(HY_THREADS), (size_t)0, HY_STREAM(stream), ROPE_ARGS(__nv_bfloat16));
#undef ROPE_ARGS
  return e == cudaSuccess ? 0 : -3;
}

// ff > 0 with ff_dst: the block row behind the last norm group also turns the feed-forward columns into relu^2.
extern "C" int b200_gate_norm(const void* y, const void* p, const float* ws, int splits, long long slab, int ld,
                              const void* w, void* dst, int dst_ld, int n_tok, int inner, int groups, float eps,
                              int ff_col, int ff, void* ff_dst, int f32, void* stream) {
  if (n_tok <= 0) return 0;
  if (groups < 1 || inner % groups || dst_ld % 4 || ff % 4 || ff_col % 4 || ld % 4 || slab % 4) return -10;
  const int gsize = inner / groups;
  const size_t smem = (size_t)gsize * sizeof(float);
  if (smem > 48 * 1024) return -10;
  dim3 grid(n_tok < 148 * 8 ? n_tok : 148 * 8, groups + (ff > 0 ? 1 : 0));
  cudaError_t e;
  if (f32) e = launch_pdl(gate_norm_kernel<float>, grid, dim3(HY_THREADS), smem, HY_STREAM(stream), (const float*)y,
                          make_proj<float>(p, ws, splits, slab, ld), (const float*)w, (float*)dst, dst_ld, n_tok, inner,
                          groups, eps, ff_col, ff, (float*)ff_dst);
  else e = launch_pdl(gate_norm_kernel<__nv_bfloat16>, grid, dim3(HY_THREADS), smem, HY_STREAM(stream),
                      (const __nv_bfloat16*)y, make_proj<__nv_bfloat16>(p, ws, splits, slab, ld), (const __nv_bfloat16*)w,
                      (__nv_bfloat16*)dst, dst_ld, n_tok, inner, groups, eps, ff_col, ff, (__nv_bfloat16*)ff_dst);
  return e == cudaSuccess ? 0 : -3;
}
