// Windowed attention of a ragged batch on tcgen05, keys and values read from the paged cache by TMA.
//
// One CTA works on one (query tile, kv head): the 128 rows of the tile are the query heads of the group times
// 128 / group consecutive tokens, so a key page is fetched once for the whole group and a tile spans few positions
// beyond its window. Key tiles are cache pages: the pages that hold the kept first tokens, then the pages of the
// window; everything between them is never touched. Two CTAs share an SM (one's page loads run under the other's
// MMAs and softmax).
//     S[128 q, 128 keys] = Q K^T   TMEM columns [0, 128);   P (bf16) overwrites columns [0, 64)
//     O[128 q, dv]      += P V     TMEM columns [128, 256)
// warp 0: TMA; warp 1: MMA issue; warps 2-5: softmax, one row per thread, in the log2 domain with a lazily moved
// reference (O is rescaled only when a row's maximum grew by more than 2^8). A sink is a row sum that starts at the
// weight of score 0. Head sizes up to 128; other sizes and fp32 take attn_ragged_kernel.
#include "proj.cuh"

namespace b200 {

struct WinParams {
  const int* cu;
  const int* start;
  const int* tile_seq;     // [n_tiles] sequence of each query tile
  const int* tile_q0;      // [n_tiles] its first token inside the portion
  const int* block_table;  // [n, max_pages]
  __nv_bfloat16* out;
  int max_pages, H, G, rep, tq;   // rep = H / G heads per group; tq tokens per tile
  int dk, dv, out_ld, window, keep, sink;
  float scale_log2;
  int* status;
};

constexpr int WIN_PAGE = 128;
struct WinSmem {
  static constexpr int Q_OFF = 0;          // 2 panels of 64 channels x 128 rows
  static constexpr int K_OFF = 32768;
  static constexpr int V_OFF = 65536;
  static constexpr int BAR_OFF = 98304;
  static constexpr int TOTAL = BAR_OFF + 256 + 1024;
};

__global__ void __launch_bounds__(192, 2)
attn_window_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_k,
                   const __grid_constant__ CUtensorMap tma_v, const WinParams p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + WinSmem::BAR_OFF);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;
  uint64_t* k_empty = bars + 2;
  uint64_t* v_full = bars + 3;
  uint64_t* v_empty = bars + 4;
  uint64_t* s_full = bars + 5;
  uint64_t* p_full = bars + 6;
  uint64_t* o_full = bars + 7;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kvh = blockIdx.x;
  const int t = gridDim.y - 1 - blockIdx.y;            // later tiles of a sequence (more keys) start first
  const int seq = p.tile_seq[t], q0 = p.tile_q0[t];
  const int row_base = p.cu[seq], len = p.cu[seq + 1] - row_base, start = p.start[seq];
  const int qlo = start + q0, qhi = start + min(q0 + p.tq, len) - 1;       // positions of the tile's tokens
  const int lo = max(0, qlo - p.window + 1);
  const int w0 = lo / WIN_PAGE, w1 = qhi / WIN_PAGE;
  const int nk = min((p.keep + WIN_PAGE - 1) / WIN_PAGE, w0);
  const int n = nk + (w1 - w0 + 1);
  const int kp = (p.dk + 63) >> 6, vp = (p.dv + 63) >> 6;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(k_full, 1);
    mbar_init(k_empty, 1);
    mbar_init(v_full, 1);
    mbar_init(v_empty, 1);
    mbar_init(s_full, 1);
    mbar_init(p_full, 4);
    mbar_init(o_full, 1);
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tm_s = *tmem_slot, tm_o = tm_s + 128;

  if (warp == 0) {
    if (lane == 0) {
      tma_prefetch_desc(&tma_k);
      tma_prefetch_desc(&tma_v);
      mbar_expect_tx(q_full, kp * p.rep * p.tq * 128);
      for (int c = 0; c < kp; ++c)
        tma_load_3d(smem + WinSmem::Q_OFF + c * 16384, &tma_q, q_full, c * 64, kvh * p.rep, row_base + q0);
      const int* bt = p.block_table + (size_t)seq * p.max_pages;
      for (int j = 0; j < n; ++j) {
        const int page = bt[j < nk ? j : w0 + (j - nk)];
        if (!mbar_wait(k_empty, (j & 1) ^ 1, p.status, ERR_TIMEOUT_EMPTY)) break;
        mbar_expect_tx(k_full, kp * 16384);
        for (int c = 0; c < kp; ++c)
          tma_load_3d(smem + WinSmem::K_OFF + c * 16384, &tma_k, k_full, c * 64, kvh, page * WIN_PAGE);
        if (!mbar_wait(v_empty, (j & 1) ^ 1, p.status, ERR_TIMEOUT_EMPTY)) break;
        mbar_expect_tx(v_full, vp * 16384);
        for (int c = 0; c < vp; ++c)
          tma_load_3d(smem + WinSmem::V_OFF + c * 16384, &tma_v, v_full, c * 64, kvh, page * WIN_PAGE);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t id_s = make_idesc_bf16(128, 128, false, false);
      const uint32_t id_o = make_idesc_bf16(128, (p.dv + 15) & ~15, false, true);
      const uint64_t dq = make_smem_desc_sw128(smem_u32(smem + WinSmem::Q_OFF), 16, 1024);
      const uint64_t dk = make_smem_desc_sw128(smem_u32(smem + WinSmem::K_OFF), 16, 1024);
      const uint64_t dv = make_smem_desc_sw128(smem_u32(smem + WinSmem::V_OFF), 16384, 1024);
      const int kn = (p.dk + 15) >> 4;
      bool ok = mbar_wait(q_full, 0, p.status, ERR_TIMEOUT_FULL);
      for (int j = 0; j < n && ok; ++j) {
        if (!mbar_wait(k_full, j & 1, p.status, ERR_TIMEOUT_FULL)) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          const uint64_t off = ((k >> 2) * 16384 + (k & 3) * 32) >> 4;
          if (k < kn) umma_bf16(tm_s, dq + off, dk + off, id_s, k > 0);   // in issue order behind P V of tile j - 1
        }
        umma_commit(s_full);
        umma_commit(k_empty);
        if (!mbar_wait(v_full, j & 1, p.status, ERR_TIMEOUT_FULL)) break;
        if (!mbar_wait(p_full, j & 1, p.status, ERR_TIMEOUT_TMEM_EMPTY)) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < 8; ++k)
          umma_bf16_ts(tm_o, tm_s + k * 8, dv + ((k * 2048) >> 4), id_o, j > 0 || k > 0);
        umma_commit(v_empty);
      }
      umma_commit(o_full);
    }
  } else {
    const int quarter = warp & 3, r = quarter * 32 + lane;
    const uint32_t lane_addr = uint32_t(quarter * 32) << 16;
    const int ti = r / p.rep, head = kvh * p.rep + r % p.rep;
    const bool row_ok = ti < p.tq && q0 + ti < len;
    const int i = min(start + q0 + ti, qhi);               // position of the row's query
    float m_ref = p.sink ? 0.f : -1e30f, l = p.sink ? 1.f : 0.f;
    bool ok = true;
    for (int j = 0; j < n; ++j) {
      if (!mbar_wait(s_full, j & 1, p.status, ERR_TIMEOUT_TMEM_FULL)) { ok = false; break; }
      tc_fence_after();
      uint32_t v[128];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32b_x32(tm_s + lane_addr + c * 32, v + c * 32);
      tmem_ld_wait();
      const int base = (j < nk ? j : w0 + (j - nk)) * WIN_PAGE;
      if (base + WIN_PAGE - 1 > qlo || base <= qhi - p.window) {          // some key of the page is hidden from some row
        const int hi_c = i - base;                          // columns up to here are not in the future
        const int lo_c = i - p.window + 1 - base;           // and from here inside the window,
        const int keep_c = p.keep - base;                   // or below this kept
#pragma unroll
        for (int c = 0; c < 128; ++c)
          if (c > hi_c || (c < lo_c && c >= keep_c)) v[c] = 0xff800000u;
      }
      float mx = -INFINITY;
#pragma unroll
      for (int c = 0; c < 128; ++c) mx = fmaxf(mx, __uint_as_float(v[c]));
      mx *= p.scale_log2;
      const bool grow = mx > m_ref + 8.f;
      const float m_new = grow ? mx : m_ref;
      const float alpha = exp2f(m_ref - m_new);
      if (j > 0 && __any_sync(0xffffffffu, grow)) {
#pragma unroll 1
        for (int c = 0; c < p.dv; c += 16) {
          uint32_t o[16];
          tmem_ld_32x32b_x16(tm_o + lane_addr + c, o);
          tmem_ld_wait();
#pragma unroll
          for (int u = 0; u < 16; ++u) o[u] = __float_as_uint(__uint_as_float(o[u]) * alpha);
          tmem_st_32x32b_x16(tm_o + lane_addr + c, o);
        }
      }
      l *= alpha;
      m_ref = m_new;
      float sum = 0.f;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int u = 0; u < 16; ++u) {
          const float e0 = exp2f(fmaf(__uint_as_float(v[c * 32 + 2 * u]), p.scale_log2, -m_ref));
          const float e1 = exp2f(fmaf(__uint_as_float(v[c * 32 + 2 * u + 1]), p.scale_log2, -m_ref));
          sum += e0 + e1;
          pk[u] = pack_bf16x2(e0, e1);
        }
        tmem_st_32x32b_x16(tm_s + lane_addr + c * 16, pk);
      }
      l += sum;
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    if (ok && mbar_wait(o_full, 0, p.status, ERR_TIMEOUT_TMEM_FULL)) {
      tc_fence_after();
      const float inv = l > 0.f ? 1.f / l : 0.f;
      __nv_bfloat16* orow = p.out + (size_t)(row_base + q0 + ti) * p.out_ld + head * p.dv;
      const bool vec = p.dv % 8 == 0;                       // out_ld is a multiple of 8
#pragma unroll 1
      for (int c = 0; c < p.dv; c += 16) {
        uint32_t o[16];
        tmem_ld_32x32b_x16(tm_o + lane_addr + c, o);
        tmem_ld_wait();
        if (!row_ok) continue;
        if (vec) {
#pragma unroll
          for (int u = 0; u < 2; ++u)
            if (c + 8 * u < p.dv) {
              uint4 w;
              w.x = pack_bf16x2(__uint_as_float(o[8 * u]) * inv, __uint_as_float(o[8 * u + 1]) * inv);
              w.y = pack_bf16x2(__uint_as_float(o[8 * u + 2]) * inv, __uint_as_float(o[8 * u + 3]) * inv);
              w.z = pack_bf16x2(__uint_as_float(o[8 * u + 4]) * inv, __uint_as_float(o[8 * u + 5]) * inv);
              w.w = pack_bf16x2(__uint_as_float(o[8 * u + 6]) * inv, __uint_as_float(o[8 * u + 7]) * inv);
              *reinterpret_cast<uint4*>(orow + c + 8 * u) = w;
            }
        } else {
#pragma unroll
          for (int u = 0; u < 16; ++u)
            if (c + u < p.dv) orow[c + u] = __float2bfloat16_rn(__uint_as_float(o[u]) * inv);
        }
      }
    }
  }

  __syncwarp();
  if (p.status != nullptr && *(volatile int*)p.status != 0) {
    // a wait gave up somewhere: give copies in flight time to land before the shared memory is released
    uint64_t t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 2000000ull) __nanosleep(1000);
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tm_s, 256);
  }
}

int make_tmap_bf16_3d(CUtensorMap* out, const void* base, uint64_t d0, uint64_t d1, uint64_t d2, uint64_t ld1, uint64_t ld2,
                      uint32_t box0, uint32_t box1, uint32_t box2);

}  // namespace b200

using namespace b200;

// bf16 q [T, H, dk_ld], caches [slots, G, dk_ld / dv_ld] with pages of 128 slots; tile_seq / tile_q0: query tiles of
// 128 / (H / G) tokens. Returns -20 for sizes the kernel does not cover.
extern "C" int b200_attn_window(const void* q, const void* k_cache, const void* v_cache, const int* cu, const int* start,
                                const int* block_table, const int* tile_seq, const int* tile_q0, int n_tiles, int T,
                                int max_pages, int num_pages, void* out, int out_ld, int H, int G, int dk, int dv,
                                int dk_ld, int dv_ld, int window, int keep, int sink, float scale, int* status,
                                void* stream) {
  if (T <= 0 || n_tiles <= 0) return 0;
  if (H % G || window < 1 || keep < 0) return -10;
  const int rep = H / G;
  if (dk > 128 || dv > 128 || dk < 1 || dv < 1 || rep > 64 || dk_ld % 8 || dv_ld % 8 || out_ld % 8 || n_tiles > 65535) return -20;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache) |
       reinterpret_cast<uintptr_t>(out)) & 15) return -12;
  const int tq = 128 / rep;
  CUtensorMap mq, mk, mv;
  int r = make_tmap_bf16_3d(&mq, q, dk, H, T, dk_ld, (uint64_t)H * dk_ld, 64, rep, tq);
  if (r) return r;
  r = make_tmap_bf16_3d(&mk, k_cache, dk, G, (uint64_t)num_pages * WIN_PAGE, dk_ld, (uint64_t)G * dk_ld, 64, 1, WIN_PAGE);
  if (r) return r;
  r = make_tmap_bf16_3d(&mv, v_cache, dv, G, (uint64_t)num_pages * WIN_PAGE, dv_ld, (uint64_t)G * dv_ld, 64, 1, WIN_PAGE);
  if (r) return r;
  static std::atomic<unsigned long long> configured{0};
  if (!set_max_smem_once(configured, attn_window_kernel, WinSmem::TOTAL)) return -2;
  WinParams p;
  p.cu = cu; p.start = start; p.tile_seq = tile_seq; p.tile_q0 = tile_q0; p.block_table = block_table;
  p.out = reinterpret_cast<__nv_bfloat16*>(out); p.max_pages = max_pages; p.H = H; p.G = G; p.rep = rep; p.tq = tq;
  p.dk = dk; p.dv = dv; p.out_ld = out_ld; p.window = window; p.keep = keep; p.sink = sink;
  p.scale_log2 = scale * 1.4426950408889634f; p.status = status;
  attn_window_kernel<<<dim3(G, n_tiles), 192, WinSmem::TOTAL, reinterpret_cast<cudaStream_t>(stream)>>>(mq, mk, mv, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
