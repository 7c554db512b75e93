// Attention of a ragged batch over a paged KV cache with a sliding window that keeps the first tokens of a sequence,
// and an optional sink (a score of 0 without a value in the softmax denominator). Query position i sees key j when
// j <= i and (i - j < window or j < keep). Every query reads its keys from the cache, the tokens of the current step
// included, so whole prompts, portions of prompts and single tokens take the same path.
#include "proj.cuh"

namespace b200 {

struct WindowArgs {
  const int* block_table;   // [n, max_pages] pages of every sequence of the batch
  int max_pages, page;
  int H, G, dk, dv, dk_ld, dv_ld, out_ld;
  int window, keep, sink;
  float scale;
};

constexpr int AW_WARPS = 8;
constexpr int AW_MAX_DV = 256;

// Any head size and either element type: one warp per (token, head), 32 keys at a time.
template <typename T>
__global__ void __launch_bounds__(AW_WARPS * 32)
attn_ragged_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache, const Ragged b,
                   T* __restrict__ out, const WindowArgs a) {
  extern __shared__ float qs_all[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* qs = qs_all + warp * a.dk;
  const long long item = blockIdx.x * (long long)AW_WARPS + warp;
  if (item >= (long long)b.T * a.H) return;
  const int t = (int)(item / a.H), h = (int)(item % a.H), g = h / (a.H / a.G);
  const int seq = b.tok_seq[t];
  const int i = b.start[seq] + (t - b.cu[seq]);          // position of the query
  const int* bt = a.block_table + (size_t)seq * a.max_pages;
  for (int c = lane; c < a.dk; c += 32) qs[c] = to_f(q[((size_t)t * a.H + h) * a.dk_ld + c]) * a.scale;
  __syncwarp();
  const int lo = i - a.window + 1 > 0 ? i - a.window + 1 : 0;
  const int kept = a.keep < lo ? a.keep : lo;            // keys [0, kept) in front of the window [lo, i]
  const int n_keys = kept + (i - lo + 1);
  float m = a.sink ? 0.f : -INFINITY, l = a.sink ? 1.f : 0.f;
  float acc[AW_MAX_DV / 32];
#pragma unroll
  for (int c = 0; c < AW_MAX_DV / 32; ++c) acc[c] = 0.f;
  for (int k0 = 0; k0 < n_keys; k0 += 32) {
    const int e = k0 + lane;
    const int j = e < kept ? e : lo + (e - kept);
    float s = -INFINITY;
    size_t slot = 0;
    if (e < n_keys) {
      slot = (size_t)bt[j / a.page] * a.page + j % a.page;
      const T* kr = k_cache + (slot * a.G + g) * a.dk_ld;
      s = 0.f;
      for (int c = 0; c < a.dk; ++c) s = fmaf(qs[c], to_f(kr[c]), s);
    }
    const float mn = fmaxf(m, warp_max(s));
    const float alpha = expf(m - mn);
    const float p = expf(s - mn);                        // 0 for lanes without a key
    l = l * alpha + warp_sum(p);
    m = mn;
#pragma unroll
    for (int c = 0; c < AW_MAX_DV / 32; ++c) acc[c] *= alpha;
    const int cnt = min(32, n_keys - k0);
    for (int e2 = 0; e2 < cnt; ++e2) {
      const float pe = __shfl_sync(0xffffffffu, p, e2);
      const long long se = __shfl_sync(0xffffffffu, (long long)slot, e2);
      const T* vr = v_cache + ((size_t)se * a.G + g) * a.dv_ld;
#pragma unroll
      for (int c = 0; c < AW_MAX_DV / 32; ++c)
        if (c * 32 + lane < a.dv) acc[c] = fmaf(pe, to_f(vr[c * 32 + lane]), acc[c]);
    }
  }
  const float inv = 1.f / l;
  T* o = out + (size_t)t * a.out_ld + h * a.dv;
#pragma unroll
  for (int c = 0; c < AW_MAX_DV / 32; ++c)
    if (c * 32 + lane < a.dv) o[c * 32 + lane] = from_f<T>(acc[c] * inv);
}

}  // namespace b200

using namespace b200;

// q [T, H, dk_ld], caches [slots, G, dk_ld / dv_ld], out rows of out_ld elements with head h at column h * dv.
extern "C" int b200_attn_ragged(const void* q, const void* k_cache, const void* v_cache, const int* cu, const int* start,
                                const int* tok_seq, const int* block_table, int n, int T, int max_pages, int page,
                                void* out, int out_ld, int H, int G, int dk, int dv, int dk_ld, int dv_ld, int window,
                                int keep, int sink, float scale, int f32, void* stream) {
  if (T <= 0 || n <= 0) return 0;
  if (H % G || dv > AW_MAX_DV || dk > 1024 || window < 1 || keep < 0) return -10;
  const Ragged b = make_ragged(cu, start, nullptr, nullptr, tok_seq, n, T);
  WindowArgs a;
  a.block_table = block_table; a.max_pages = max_pages; a.page = page; a.H = H; a.G = G; a.dk = dk; a.dv = dv;
  a.dk_ld = dk_ld; a.dv_ld = dv_ld; a.out_ld = out_ld; a.window = window; a.keep = keep; a.sink = sink; a.scale = scale;
  const long long blocks = ((long long)T * H + AW_WARPS - 1) / AW_WARPS;
  const size_t smem = sizeof(float) * AW_WARPS * dk;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (f32)
    attn_ragged_kernel<float><<<(unsigned)blocks, AW_WARPS * 32, smem, st>>>((const float*)q, (const float*)k_cache,
                                                                             (const float*)v_cache, b, (float*)out, a);
  else
    attn_ragged_kernel<__nv_bfloat16><<<(unsigned)blocks, AW_WARPS * 32, smem, st>>>(
        (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_cache, (const __nv_bfloat16*)v_cache, b, (__nv_bfloat16*)out, a);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
