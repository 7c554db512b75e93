// Mamba-2 (state-space duality) mixer kernels over a ragged batch: causal convolution with carried taps, the
// recurrence token by token (any size, bf16 or all-fp32), and the fused decode step. Per head h of a group g
//     S_t = exp(-exp(A_log_h) dt_t) S_(t-1) + dt_t B_t x_t^T      (S is [N, P], kept in fp32)
//     y_t = S_t^T C_t + D_h x_t
// Input projection columns: [z: inner | x: inner | B: G N | C: G N | dt: H]; x, B and C pass the convolution.
//
// The convolution's history is a ring of `taps` entries per state row: the input of position p sits in entry
// p mod taps. A decode step writes entry p mod taps (position p - taps, no longer needed) and reads the others, so the
// blocks of one launch may read and write the ring of the same row without ordering.
#include "proj.cuh"

namespace b200 {

struct SsdDims {
  int H, P, N, G, taps;
  int inner, cc;      // H P; channels of the convolution: inner + 2 G N
};

// Convolution input of position `ps` of a sequence for channel column c: this step's projection when the token is part
// of the portion (offset o >= 0), the ring for earlier positions, zero before the start of the sequence.
template <typename T, int V>
__device__ __forceinline__ void conv_input(const Proj<T>& src, const T* __restrict__ ring, int row0, int o, int start,
                                           int taps, int cc, int xcol, int c, float* f) {
  if (o >= 0) {
    if (V == 4) src.get4(row0 + o, xcol + c, f);
    else f[0] = src.get(row0 + o, xcol + c);
    return;
  }
  const int ps = start + o;
  if (ps < 0) {
#pragma unroll
    for (int k = 0; k < V; ++k) f[k] = 0.f;
    return;
  }
  const T* r = ring + (size_t)(ps % taps) * cc + c;
  if (V == 4) load4(r, f);
  else f[0] = to_f(r[0]);
}

// out[t, c] = silu(bias[c] + sum_k w[c, k] u[t - taps + 1 + k, c]); dt[t, h] = softplus(proj + dt_bias[h])
template <typename T, int V>
__global__ void __launch_bounds__(256)
conv_kernel(const Proj<T> src, const Ragged b, const T* __restrict__ ring, const T* __restrict__ w,
            const T* __restrict__ bias, const T* __restrict__ dt_bias, T* __restrict__ out, float* __restrict__ dt,
            const SsdDims d) {
  const int nv = d.cc / V;
  const int per_tok = nv + d.H;
  const long long total = (long long)b.T * per_tok;
  for (long long idx = blockIdx.x * (long long)blockDim.x + threadIdx.x; idx < total;
       idx += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(idx / per_tok), e = (int)(idx % per_tok);
    if (e >= nv) {
      const int h = e - nv;
      dt[(size_t)h * b.T + t] = softplus_f(src.get_raw(t, d.inner + d.cc + h) + to_f(dt_bias[h]));
      continue;
    }
    const int c = e * V;
    const int i = b.tok_seq[t];
    const int row0 = b.cu[i], start = b.start[i], o = t - row0;
    const T* rg = ring + (size_t)b.row[i] * d.taps * d.cc;
    float acc[V];
#pragma unroll
    for (int k = 0; k < V; ++k) acc[k] = to_f(bias[c + k]);
    for (int k = 0; k < d.taps; ++k) {
      float u[V];
      conv_input<T, V>(src, rg, row0, o - (d.taps - 1 - k), start, d.taps, d.cc, d.inner, c, u);
#pragma unroll
      for (int q = 0; q < V; ++q) acc[q] = fmaf(to_f(w[(size_t)(c + q) * d.taps + k]), u[q], acc[q]);
    }
#pragma unroll
    for (int q = 0; q < V; ++q) acc[q] = silu_f(acc[q]);
    T* dst = out + (size_t)t * d.cc + c;
    if (V == 4) store4(dst, acc);
    else dst[0] = from_f<T>(acc[0]);
  }
}

// The same for long batches: a thread slides down a run of tokens with the last TAPS - 1 inputs of its four channels in
// registers, so every input is read once (and TAPS - 1 once more per run). A run may cross into another sequence.
constexpr int CONV_RUN = 32, CONV_BATCH = 4;
template <typename T, int TAPS>
__global__ void __launch_bounds__(128, 6)
conv_run_kernel(const Proj<T> src, const Ragged b, const T* __restrict__ ring, const T* __restrict__ w,
                const T* __restrict__ bias, T* __restrict__ out, const SsdDims d) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (c >= d.cc) return;
  const int t0 = blockIdx.y * CONV_RUN, t1 = min(b.T, t0 + CONV_RUN);
  float wt[TAPS][4], bs[4], hist[TAPS][4];
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    bs[q] = to_f(bias[c + q]);
#pragma unroll
    for (int k = 0; k < TAPS; ++k) wt[k][q] = to_f(w[(size_t)(c + q) * TAPS + k]);
  }
  int seq = -1;
  for (int t = t0; t < t1; t += CONV_BATCH) {
    float u[CONV_BATCH][4];
    int ids[CONV_BATCH];
#pragma unroll
    for (int j = 0; j < CONV_BATCH; ++j)
      if (t + j < t1) {
        load4(src.p + (size_t)(t + j) * src.ld + d.inner + c, u[j]);
        ids[j] = b.tok_seq[t + j];
      }
#pragma unroll
    for (int j = 0; j < CONV_BATCH; ++j) {
      if (t + j >= t1) break;
      const int i = ids[j];
      if (i != seq) {                                     // the run's first token, or another sequence begins
        seq = i;
        const int row0 = b.cu[i], o = t + j - row0;
#pragma unroll
        for (int k = 1; k < TAPS; ++k)
          conv_input<T, 4>(src, ring + (size_t)b.row[i] * d.taps * d.cc, row0, o - (TAPS - k), b.start[i], TAPS, d.cc,
                           d.inner, c, hist[k]);          // hist[k]: the input TAPS - k tokens back
      }
      float acc[4];
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        acc[q] = bs[q];
#pragma unroll
        for (int k = 1; k < TAPS; ++k) acc[q] = fmaf(wt[k - 1][q], hist[k][q], acc[q]);
        acc[q] = silu_f(fmaf(wt[TAPS - 1][q], u[j][q], acc[q]));
#pragma unroll
        for (int k = 1; k + 1 < TAPS; ++k) hist[k][q] = hist[k + 1][q];
        if (TAPS > 1) hist[TAPS - 1][q] = u[j][q];
      }
      store4(out + (size_t)(t + j) * d.cc + c, acc);
    }
  }
}

// dt[h, t] = softplus(proj + dt_bias[h]) for the run kernel: 32 tokens per block, written in whole lines.
template <typename T>
__global__ void __launch_bounds__(256)
dt_kernel(const Proj<T> src, const T* __restrict__ dt_bias, float* __restrict__ dt, int n_tok, const SsdDims d) {
  const int t = blockIdx.x * 32 + (threadIdx.x & 31);
  if (t >= n_tok) return;
  for (int h = threadIdx.x >> 5; h < d.H; h += 8)
    dt[(size_t)h * n_tok + t] = softplus_f(src.get_raw(t, d.inner + d.cc + h) + to_f(dt_bias[h]));
}

// The last taps - 1 inputs of every portion go to the ring (after conv_kernel has read the old entries).
template <typename T>
__global__ void conv_ring_kernel(const Proj<T> src, const Ragged b, T* __restrict__ ring, const SsdDims d) {
  const int i = blockIdx.y;
  if (!b.live(i)) return;
  const int row0 = b.cu[i], len = b.cu[i + 1] - row0, start = b.start[i];
  T* rg = ring + (size_t)b.row[i] * d.taps * d.cc;
  for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < d.cc; c += gridDim.x * blockDim.x)
    for (int o = max(0, len - (d.taps - 1)); o < len; ++o)
      rg[(size_t)((start + o) % d.taps) * d.cc + c] = from_f<T>(src.get(row0 + o, d.inner + c));
}

// Token-by-token recurrence of one (sequence, head) per block, the state in shared memory.
template <typename T>
__global__ void __launch_bounds__(256)
ssd_scan_kernel(const T* __restrict__ xbc, const float* __restrict__ dt, const Ragged b, const T* __restrict__ a_log,
                const T* __restrict__ dskip, float* __restrict__ state, T* __restrict__ y, const SsdDims d) {
  extern __shared__ float sm[];
  float* s = sm;                       // [N, P]
  float* sb = s + d.N * d.P;           // [N]
  float* sc = sb + d.N;                // [N]
  float* sx = sc + d.N;                // [P]
  float* part = sx + d.P;              // [groups of n, P]
  const int h = blockIdx.x, i = blockIdx.y;
  const int row0 = b.cu[i], len = b.cu[i + 1] - row0;
  if (len <= 0) return;
  const int g = h / (d.H / d.G);
  const int ng = blockDim.x / d.P, pg = threadIdx.x / d.P, p = threadIdx.x % d.P;
  const int nper = (d.N + ng - 1) / ng, n0 = pg * nper, n1 = pg < ng ? min(d.N, n0 + nper) : n0;
  float* gs = state + ((size_t)b.row[i] * d.H + h) * d.N * d.P;
  const bool fresh = b.start[i] == 0;
  for (int k = threadIdx.x; k < d.N * d.P; k += blockDim.x) s[k] = fresh ? 0.f : gs[k];
  const float a = -expf(to_f(a_log[h])), dk = to_f(dskip[h]);
  for (int o = 0; o < len; ++o) {
    const T* r = xbc + (size_t)(row0 + o) * d.cc;
    __syncthreads();
    for (int k = threadIdx.x; k < d.N; k += blockDim.x) {
      sb[k] = to_f(r[d.inner + g * d.N + k]);
      sc[k] = to_f(r[d.inner + (d.G + g) * d.N + k]);
    }
    for (int k = threadIdx.x; k < d.P; k += blockDim.x) sx[k] = to_f(r[h * d.P + k]);
    const float dtv = dt[(size_t)h * b.T + row0 + o];
    const float decay = expf(a * dtv);
    __syncthreads();
    if (pg < ng) {
      const float xd = dtv * sx[p];
      float acc = 0.f;
      for (int n = n0; n < n1; ++n) {
        const float v = fmaf(decay, s[n * d.P + p], xd * sb[n]);
        s[n * d.P + p] = v;
        acc = fmaf(v, sc[n], acc);
      }
      part[pg * d.P + p] = acc;
    }
    __syncthreads();
    for (int k = threadIdx.x; k < d.P; k += blockDim.x) {
      float acc = dk * sx[k];
      for (int q = 0; q < ng; ++q) acc += part[q * d.P + k];
      y[(size_t)(row0 + o) * d.inner + h * d.P + k] = from_f<T>(acc);
    }
  }
  __syncthreads();
  if (b.live(i))
    for (int k = threadIdx.x; k < d.N * d.P; k += blockDim.x) gs[k] = s[k];
}

// One token per sequence: convolution, step size, state update and read-out of one (head, sequence) per block. The
// state streams through registers once (V channels per access); bound by its bytes.
template <typename T, int V>
__global__ void __launch_bounds__(128)
ssd_decode_kernel(const Proj<T> src, const Ragged b, T* __restrict__ ring, const T* __restrict__ w,
                  const T* __restrict__ bias, const T* __restrict__ dt_bias, const T* __restrict__ a_log,
                  const T* __restrict__ dskip, float* __restrict__ state, T* __restrict__ y, const SsdDims d) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];
  float* sx = sm;                      // [P]
  float* sb = sx + ((d.P + 3) & ~3);   // [N]
  float* sc = sb + d.N;                // [N]
  float* part = sc + d.N;              // [threads / lanes of a row, P]
  const int h = blockIdx.x, i = blockIdx.y;
  if (!b.live(i)) {                    // keeps whatever reads the row finite, and every state untouched
    for (int p = threadIdx.x; p < d.P; p += blockDim.x) y[(size_t)i * d.inner + h * d.P + p] = from_f<T>(0.f);
    return;
  }
  const int hpg = d.H / d.G, g = h / hpg;
  const int pos = b.start[i];
  T* rg = ring + (size_t)b.row[i] * d.taps * d.cc;
  const bool owns_bc = h == g * hpg;
  for (int e = threadIdx.x; e < d.P + 2 * d.N; e += blockDim.x) {
    const int c = e < d.P ? h * d.P + e
                          : (e < d.P + d.N ? d.inner + g * d.N + (e - d.P) : d.inner + (d.G + g) * d.N + (e - d.P - d.N));
    const float cur = src.get(i, d.inner + c);
    float acc = fmaf(to_f(w[(size_t)c * d.taps + d.taps - 1]), cur, to_f(bias[c]));
    for (int k = 0; k < d.taps - 1; ++k) {
      const int ps = pos - (d.taps - 1 - k);
      if (ps >= 0) acc = fmaf(to_f(w[(size_t)c * d.taps + k]), to_f(rg[(size_t)(ps % d.taps) * d.cc + c]), acc);
    }
    if (e < d.P || owns_bc) rg[(size_t)(pos % d.taps) * d.cc + c] = from_f<T>(cur);
    const float v = round_to<T>(silu_f(acc));
    if (e < d.P) sx[e] = v;
    else sb[e - d.P] = v;              // B, then C (sc follows sb)
  }
  const float dtv = softplus_f(src.get_raw(i, d.inner + d.cc + h) + to_f(dt_bias[h]));
  const float decay = expf(-expf(to_f(a_log[h])) * dtv), dk = to_f(dskip[h]);
  const bool fresh = pos == 0;
  float* gs = state + ((size_t)b.row[i] * d.H + h) * d.N * d.P;
  const int lanes = d.P / V;           // threads across one row of the state
  const int ng = blockDim.x / lanes, pg = threadIdx.x / lanes, p = (threadIdx.x % lanes) * V;
  __syncthreads();
  if (pg < ng) {
    float xd[V], acc[V];
#pragma unroll
    for (int k = 0; k < V; ++k) { xd[k] = dtv * sx[p + k]; acc[k] = 0.f; }
#pragma unroll 8
    for (int n = pg; n < d.N; n += ng) {
      float f[V];
      float* q = gs + (size_t)n * d.P + p;
      if (fresh) {
#pragma unroll
        for (int k = 0; k < V; ++k) f[k] = 0.f;
      } else if (V == 4) {
        load4(q, f);
      } else {
        f[0] = q[0];
      }
#pragma unroll
      for (int k = 0; k < V; ++k) {
        f[k] = fmaf(decay, f[k], xd[k] * sb[n]);
        acc[k] = fmaf(f[k], sc[n], acc[k]);
      }
      if (V == 4) store4(q, f);
      else q[0] = f[0];
    }
#pragma unroll
    for (int k = 0; k < V; ++k) part[pg * d.P + p + k] = acc[k];
  }
  __syncthreads();
  for (int k = threadIdx.x; k < d.P; k += blockDim.x) {
    float acc = dk * sx[k];
    for (int q = 0; q < ng; ++q) acc += part[q * d.P + k];
    y[(size_t)i * d.inner + h * d.P + k] = from_f<T>(acc);
  }
}

static int ssd_dims(SsdDims& d, int H, int P, int N, int G, int taps) {
  if (H < 1 || P < 1 || N < 1 || G < 1 || H % G || taps < 1) return -10;
  d.H = H; d.P = P; d.N = N; d.G = G; d.taps = taps; d.inner = H * P; d.cc = d.inner + 2 * G * N;
  return 0;
}

template <typename T>
static int launch_conv(const Proj<T>& src, const Ragged& b, T* ring, const T* w, const T* bias, const T* dt_bias, T* out,
                       float* dt, const SsdDims& d, cudaStream_t st) {
  const bool vec = d.cc % 4 == 0 && d.inner % 4 == 0 && src.ld % 4 == 0 && src.slab % 4 == 0;
  if (vec && src.ws == nullptr && b.T >= 64 && d.taps >= 1 && d.taps <= 4) {
    const dim3 grid((d.cc / 4 + 127) / 128, (b.T + CONV_RUN - 1) / CONV_RUN);
    if (grid.y > 65535) return -10;
    if (d.taps == 1) conv_run_kernel<T, 1><<<grid, 128, 0, st>>>(src, b, ring, w, bias, out, d);
    else if (d.taps == 2) conv_run_kernel<T, 2><<<grid, 128, 0, st>>>(src, b, ring, w, bias, out, d);
    else if (d.taps == 3) conv_run_kernel<T, 3><<<grid, 128, 0, st>>>(src, b, ring, w, bias, out, d);
    else conv_run_kernel<T, 4><<<grid, 128, 0, st>>>(src, b, ring, w, bias, out, d);
    dt_kernel<T><<<(b.T + 31) / 32, 256, 0, st>>>(src, dt_bias, dt, b.T, d);
    if (cudaGetLastError() != cudaSuccess) return -3;
    if (d.taps > 1) conv_ring_kernel<T><<<dim3((d.cc + 255) / 256, b.n), 256, 0, st>>>(src, b, ring, d);
    return cudaGetLastError() == cudaSuccess ? 0 : -3;
  }
  const long long work = (long long)b.T * ((vec ? d.cc / 4 : d.cc) + d.H);
  long long blocks = (work + 255) / 256;
  if (blocks > 148 * 32) blocks = 148 * 32;
  if (vec) conv_kernel<T, 4><<<(int)blocks, 256, 0, st>>>(src, b, ring, w, bias, dt_bias, out, dt, d);
  else conv_kernel<T, 1><<<(int)blocks, 256, 0, st>>>(src, b, ring, w, bias, dt_bias, out, dt, d);
  if (cudaGetLastError() != cudaSuccess) return -3;
  if (d.taps > 1) conv_ring_kernel<T><<<dim3((d.cc + 255) / 256, b.n), 256, 0, st>>>(src, b, ring, d);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

}  // namespace b200

using namespace b200;
#define SSD_STREAM(s) reinterpret_cast<cudaStream_t>(s)

// Causal convolution + silu of a ragged batch, step sizes, and the ring update. out [T, cc], dt fp32 [H, T].
extern "C" int b200_ssd_conv(const void* p, const float* ws, int splits, long long slab, int ld, const int* cu,
                             const int* start, const int* row, const int* active, const int* tok_seq, int n, int T,
                             void* ring, const void* w, const void* bias, const void* dt_bias, void* out, float* dt, int H,
                             int P, int N, int G, int taps, int f32, void* stream) {
  if (T <= 0 || n <= 0) return 0;
  SsdDims d;
  if (int r = ssd_dims(d, H, P, N, G, taps)) return r;
  if (n > 65535) return -10;
  const Ragged b = make_ragged(cu, start, row, active, tok_seq, n, T);
  if (f32)
    return launch_conv<float>(make_proj<float>(p, ws, splits, slab, ld), b, (float*)ring, (const float*)w,
                              (const float*)bias, (const float*)dt_bias, (float*)out, dt, d, SSD_STREAM(stream));
  typedef __nv_bfloat16 B16;
  return launch_conv<B16>(make_proj<B16>(p, ws, splits, slab, ld), b, (B16*)ring, (const B16*)w, (const B16*)bias,
                          (const B16*)dt_bias, (B16*)out, dt, d, SSD_STREAM(stream));
}

// Token-by-token scan of a ragged batch; reads and writes the fp32 state rows [*, H, N, P]. y [T, inner].
extern "C" int b200_ssd_scan(const void* xbc, const float* dt, const int* cu, const int* start, const int* row,
                             const int* active, const int* tok_seq, int n, int T, const void* a_log, const void* dskip,
                             float* state, void* y, int H, int P, int N, int G, int taps, int f32, void* stream) {
  if (T <= 0 || n <= 0) return 0;
  SsdDims d;
  if (int r = ssd_dims(d, H, P, N, G, taps)) return r;
  if (P > 256 || n > 65535) return -10;
  const int ng = 256 / P;
  const size_t smem = sizeof(float) * ((size_t)N * P + 2 * N + P + (size_t)ng * P);
  if (smem > 200 * 1024) return -10;
  const Ragged b = make_ragged(cu, start, row, active, tok_seq, n, T);
  const dim3 grid(H, n);
  static std::atomic<unsigned long long> cf{0}, cb{0};
  if (f32) {
    if (!set_max_smem_once(cf, ssd_scan_kernel<float>, 200 * 1024)) return -2;
    ssd_scan_kernel<float><<<grid, 256, smem, SSD_STREAM(stream)>>>((const float*)xbc, dt, b, (const float*)a_log,
                                                                    (const float*)dskip, state, (float*)y, d);
  } else {
    typedef __nv_bfloat16 B16;
    if (!set_max_smem_once(cb, ssd_scan_kernel<B16>, 200 * 1024)) return -2;
    ssd_scan_kernel<B16><<<grid, 256, smem, SSD_STREAM(stream)>>>((const B16*)xbc, dt, b, (const B16*)a_log,
                                                                  (const B16*)dskip, state, (B16*)y, d);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}

// Decode step of `n` sequences (one token each, row i of the projection). y [n, inner].
extern "C" int b200_ssd_decode(const void* p, const float* ws, int splits, long long slab, int ld, const int* start,
                               const int* row, const int* active, int n, void* ring, const void* w, const void* bias,
                               const void* dt_bias, const void* a_log, const void* dskip, float* state, void* y, int H,
                               int P, int N, int G, int taps, int f32, void* stream) {
  if (n <= 0) return 0;
  SsdDims d;
  if (int r = ssd_dims(d, H, P, N, G, taps)) return r;
  const bool vec = P % 4 == 0;
  const int lanes = vec ? P / 4 : P;
  if (lanes > 128 || n > 65535) return -10;
  const int ng = 128 / lanes;
  const size_t smem = sizeof(float) * ((size_t)((P + 3) & ~3) + 2 * N + (size_t)ng * P);
  if (smem > 48 * 1024) return -10;
  const Ragged b = make_ragged(nullptr, start, row, active, nullptr, n, n);
  const dim3 grid(H, n);
#define DEC_ARGS(TT)                                                                                                   \
  make_proj<TT>(p, ws, splits, slab, ld), b, (TT*)ring, (const TT*)w, (const TT*)bias, (const TT*)dt_bias,             \
      (const TT*)a_log, (const TT*)dskip, state, (TT*)y, d
  cudaError_t e;
  cudaStream_t st = SSD_STREAM(stream);
  if (f32) e = vec ? launch_pdl(ssd_decode_kernel<float, 4>, grid, dim3(128), smem, st, DEC_ARGS(float))
                   : launch_pdl(ssd_decode_kernel<float, 1>, grid, dim3(128), smem, st, DEC_ARGS(float));
  else e = vec ? launch_pdl(ssd_decode_kernel<__nv_bfloat16, 4>, grid, dim3(128), smem, st, DEC_ARGS(__nv_bfloat16))
               : launch_pdl(ssd_decode_kernel<__nv_bfloat16, 1>, grid, dim3(128), smem, st, DEC_ARGS(__nv_bfloat16));
#undef DEC_ARGS
  return e == cudaSuccess ? 0 : -3;
}
