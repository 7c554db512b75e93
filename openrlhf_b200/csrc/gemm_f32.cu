// True fp32 GEMM for the 32-bit serving mode: C[M,N] (+)= A[M,K] W[N,K]^T on the FMA pipe, no reduced-precision tensor
// mode anywhere. 64 x 64 tiles, 256 threads, 4 x 4 accumulators per thread; ragged edges in every dimension.
#include "proj.cuh"

namespace b200 {

constexpr int F32_T = 64, F32_K = 16;

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ A, const float* __restrict__ W, float* __restrict__ C, int M, int N, int K,
                int lda, int ldw, int ldc, int accumulate) {
  __shared__ float sa[F32_K][F32_T + 4], sw[F32_K][F32_T + 4];
  const int m0 = blockIdx.y * F32_T, n0 = blockIdx.x * F32_T;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += F32_K) {
    for (int i = threadIdx.x; i < F32_T * F32_K; i += 256) {
      const int r = i / F32_K, k = i % F32_K;
      sa[k][r] = (m0 + r < M && k0 + k < K) ? A[(size_t)(m0 + r) * lda + k0 + k] : 0.f;
      sw[k][r] = (n0 + r < N && k0 + k < K) ? W[(size_t)(n0 + r) * ldw + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < F32_K; ++k) {
      float a[4], w[4];
      load4(&sa[k][ty * 4], a);
      load4(&sw[k][tx * 4], w);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < N) {
        float* c = C + (size_t)m * ldc + n;
        *c = accumulate ? *c + acc[i][j] : acc[i][j];
      }
    }
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_gemm_f32(const float* A, const float* W, float* C, int M, int N, int K, int lda, int ldw, int ldc,
                             int accumulate, void* stream) {
  if (M <= 0 || N <= 0) return 0;
  dim3 grid((N + F32_T - 1) / F32_T, (M + F32_T - 1) / F32_T);
  if (grid.y > 65535) return -10;
  gemm_f32_kernel<<<grid, 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(A, W, C, M, N, K, lda, ldw, ldc, accumulate);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
