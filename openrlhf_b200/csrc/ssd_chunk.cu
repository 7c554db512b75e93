// Mamba-2 scan of whole portions on tcgen05: 128 tokens at a time, the state of a head resident in tensor memory.
//
// One CTA walks the chunks of one (sequence, head); two CTAs share an SM, so that one's loads and elementwise work run
// under the other's MMAs. With cum_t = sum of a dt over the chunk up to t (a = -exp(A_log)), per chunk
//     G = C B^T                                   [128 t, 128 s]   A, B: smem K-major
//     Y = C S                                     [128 t, 64 p]    B: S, smem MN-major (hi + lo)
//     Y = e^{cum_t} Y + M X,  M_ts = G_ts e^{cum_t - cum_s} dt_s (s <= t)   A: M in TMEM (hi + lo), B: X smem MN-major
//     S = e^{cum_end} S + B^T Xw,  Xw_t = x_t e^{cum_end - cum_t} dt_t      A: B smem MN-major, B: Xw smem (hi + lo)
// B, C and x are bf16 activations. Everything else that enters a product (the state, the decay-weighted scores, the
// weighted inputs) is a 32-bit quantity: it is split into a bf16 high part and a bf16 remainder and multiplied twice,
// and the state itself stays fp32 in TMEM from the first chunk to the last.
//
// TMEM columns: [0, 128) G, then M (hi | lo); [128, 192) Y; [192, 256) S (lane = state row n).
// Warps 0-7: a token row (or state row) per thread, half of the columns each. Warp 8: TMA and MMA issue.
#include "proj.cuh"

namespace b200 {

int make_tmap_bf16_2d(CUtensorMap* out, const void* base, uint64_t rows, uint64_t cols, uint64_t ld, uint32_t box_rows,
                      uint32_t box_cols);

struct SsdChunkParams {
  const float* dt;            // [H, T] after softplus
  const __nv_bfloat16* a_log;
  const __nv_bfloat16* dskip;
  float* state;               // [rows, H, N, P]
  __nv_bfloat16* y;           // [T, inner]
  Ragged b;
  int H, P, N, G, inner;
  int pblocks;                // ceil(P / 64)
  // long portions on few heads: segments of seg_chunks chunks run side by side (0: one CTA walks the whole portion).
  // seg_state [n, H, n_seg, N, P] and seg_log2 [n, H, n_seg] hold every segment's own contribution to the state and its
  // summed log2 decay after the first pass, the state at its start after the combination
  int seg_chunks, n_seg;
  float* seg_state;
  float* seg_log2;
  int* status;
};

constexpr int SC_Q = 128;               // tokens per chunk
constexpr int SC_PB = 64;               // channels of x per CTA
struct ScSmem {
  static constexpr int B_OFF = 0;               // 2 panels of 64 columns x 128 rows
  static constexpr int C_OFF = 32768;           // likewise; refilled for the next chunk once G and C S are computed
  static constexpr int X_OFF = 65536;           // 1 panel; then the chunk's y on its way out
  static constexpr int S_OFF = 81920;           // S as bf16 hi, lo: 128 rows (n) of 64 channels each; then Xw, hi, lo
  static constexpr int W_OFF = 114688;          // [128] weight of token s in the rows behind its block
  static constexpr int BAR_OFF = W_OFF + 512;
  static constexpr int TOTAL = BAR_OFF + 512;   // 113 KB: two CTAs per SM
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two values -> packed bf16 high parts (truncated: the upper halves of the words) and packed bf16 remainders
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  const uint32_t ua = __float_as_uint(a), ub = __float_as_uint(b);
  hi = __byte_perm(ua, ub, 0x7632);
  lo = pack_bf16x2(a - __uint_as_float(ua & 0xffff0000u), b - __uint_as_float(ub & 0xffff0000u));
}
// byte offset of 16-byte piece j of row r in a tile of 128-byte rows with the 128-byte swizzle
__device__ __forceinline__ int sw128(int r, int j) { return r * 128 + ((j ^ (r & 7)) << 4); }

// STATE_ONLY: the first pass over segments; only the recurrence runs (from zero), nothing is read out.
template <bool STATE_ONLY>
__global__ void __launch_bounds__(288, 2)
ssd_chunk_kernel(const __grid_constant__ CUtensorMap tma, const SsdChunkParams p) {
  extern __shared__ __align__(1024) uint8_t smem[];
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + ScSmem::BAR_OFF);
  uint64_t* full = bars;            // the chunk's B tile has landed (c_full, x_full: C, x)
  uint64_t* s_ready = bars + 1;     // S split into smem, decayed in TMEM
  uint64_t* g_full = bars + 2;      // G and C S are in TMEM
  uint64_t* m_ready = bars + 3;     // M in TMEM, Y scaled
  uint64_t* xw_ready = bars + 4;    // Xw in smem
  uint64_t* done = bars + 5;        // Y and S of the chunk are in TMEM, all tiles free
  uint64_t* c_full = bars + 6;
  uint64_t* x_full = bars + 7;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 8);
  float* wtot = reinterpret_cast<float*>(bars + 10);      // [4] warp totals
  float* wsm = reinterpret_cast<float*>(smem + ScSmem::W_OFF);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, seq = blockIdx.y, p0 = (blockIdx.z % p.pblocks) * SC_PB, seg = blockIdx.z / p.pblocks;
  int row0 = p.b.cu[seq], len = p.b.cu[seq + 1] - row0;
  bool last = true;                     // the CTA that ends the portion
  if (p.seg_chunks > 0) {
    const int off = seg * p.seg_chunks * SC_Q;
    row0 += off;
    len -= off;
    last = len <= p.seg_chunks * SC_Q;
    len = min(len, p.seg_chunks * SC_Q);
  }
  if (len <= 0 || (STATE_ONLY && last)) return;         // the last segment's contribution is nobody's start
  if (smem_u32(smem) & 1023) {          // the swizzled tiles need 1024-byte alignment; there is no room for slack
    if (threadIdx.x == 0 && p.status != nullptr) atomicCAS(p.status, 0, ERR_BAD_ARG);
    return;
  }
  const int n_chunks = (len + SC_Q - 1) / SC_Q;
  const int g = h / (p.H / p.G);
  const int panels = (p.N + 63) >> 6;

  if (threadIdx.x == 0) {
    mbar_init(full, 1);
    mbar_init(c_full, 1);
    mbar_init(x_full, 1);
    mbar_init(s_ready, 8);
    mbar_init(g_full, 1);
    mbar_init(m_ready, 8);
    mbar_init(xw_ready, 8);
    mbar_init(done, 1);
    mbar_fence_init();
  }
  if (warp == 8) {
    tmem_alloc(tmem_slot, 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t tm_g = tmem, tm_y = tmem + 128, tm_s = tmem + 192;

  if (warp == 8) {
    if (lane == 0) {
      constexpr uint32_t id_g = make_idesc_bf16(128, 128, false, false);
      constexpr uint32_t id_y = make_idesc_bf16(128, SC_PB, false, true);
      constexpr uint32_t id_s = make_idesc_bf16(128, SC_PB, true, true);
      const uint32_t sb = smem_u32(smem + ScSmem::B_OFF), sc = smem_u32(smem + ScSmem::C_OFF);
      const uint32_t sx = smem_u32(smem + ScSmem::X_OFF), ss = smem_u32(smem + ScSmem::S_OFF);
      tma_prefetch_desc(&tma);
      auto load_c = [&](int c) {
        mbar_expect_tx(c_full, panels * 16384);
        for (int q = 0; q < panels; ++q)
          tma_load_2d(smem + ScSmem::C_OFF + q * 16384, &tma, c_full, p.inner + (p.G + g) * p.N + q * 64, row0 + c * SC_Q);
      };
      auto load_b = [&](int c) {
        mbar_expect_tx(full, panels * 16384);
        for (int q = 0; q < panels; ++q)
          tma_load_2d(smem + ScSmem::B_OFF + q * 16384, &tma, full, p.inner + g * p.N + q * 64, row0 + c * SC_Q);
      };
      load_b(0);
      if (!STATE_ONLY) load_c(0);
      const int kn = p.N >> 4;
      // descriptors of the first K step; a step adds its byte offset / 16 to the address field
      const uint64_t c_k = make_smem_desc_sw128(sc, 16, 1024), b_k = make_smem_desc_sw128(sb, 16, 1024);
      const uint64_t b_mn = make_smem_desc_sw128(sb, 16384, 1024), x_mn = make_smem_desc_sw128(sx, 16384, 1024);
      const uint64_t s_mn = make_smem_desc_sw128(ss, 16384, 1024);
      for (int c = 0; c < n_chunks; ++c) {
        const uint32_t ph = c & 1;
        if (!mbar_wait(full, ph, p.status, ERR_TIMEOUT_FULL)) break;
        if (!STATE_ONLY && !mbar_wait(c_full, ph, p.status, ERR_TIMEOUT_FULL)) break;
        tc_fence_after();
#pragma unroll
        for (int k = 0; k < 8; ++k) {
          const uint64_t off = ((k >> 2) * 16384 + (k & 3) * 32) >> 4;
          if (!STATE_ONLY && k < kn) umma_bf16(tm_g, c_k + off, b_k + off, id_g, k > 0);
        }
        if (!mbar_wait(s_ready, ph, p.status, ERR_TIMEOUT_TMEM_EMPTY)) break;
        tc_fence_after();
        mbar_expect_tx(x_full, 16384);          // the previous chunk's y, staged in this tile, has been copied out
        tma_load_2d(smem + ScSmem::X_OFF, &tma, x_full, h * p.P + p0, row0 + c * SC_Q);
        if (!STATE_ONLY) {
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            const int k = i & 7;
            const uint64_t off = ((k >> 2) * 16384 + (k & 3) * 32) >> 4;
            if (k < kn) umma_bf16(tm_y, c_k + off, s_mn + (((i >> 3) * 16384 + k * 2048) >> 4), id_y, i > 0);
          }
          umma_commit(g_full);
          if (c + 1 < n_chunks) {
            if (!mbar_wait(g_full, ph, p.status, ERR_TIMEOUT_EMPTY)) break;
            load_c(c + 1);
          }
        }
        if (!mbar_wait(x_full, ph, p.status, ERR_TIMEOUT_FULL)) break;
        if (!STATE_ONLY) {
          if (!mbar_wait(m_ready, ph, p.status, ERR_TIMEOUT_TMEM_EMPTY)) break;
          tc_fence_after();
#pragma unroll
          for (int i = 0; i < 16; ++i)
            umma_bf16_ts(tm_y, tm_g + (i >> 3) * 64 + (i & 7) * 8, x_mn + (((i & 7) * 2048) >> 4), id_y, 1u);
        }
        if (!mbar_wait(xw_ready, ph, p.status, ERR_TIMEOUT_TMEM_EMPTY)) break;
        tc_fence_after();
#pragma unroll
        for (int i = 0; i < 16; ++i)
          umma_bf16(tm_s, b_mn + (((i & 7) * 2048) >> 4), s_mn + (((i >> 3) * 16384 + (i & 7) * 2048) >> 4), id_s, 1u);
        umma_commit(done);
        if (c + 1 < n_chunks) {
          if (!mbar_wait(done, ph, p.status, ERR_TIMEOUT_EMPTY)) break;
          load_b(c + 1);
        }
      }
    }
  } else {
    // warps w and w + 4 share a lane quarter: the same 32 rows, half of the columns each
    const int half = warp >> 2, quarter = warp & 3;
    const int t = quarter * 32 + lane;                      // token of the chunk, and state row
    const uint32_t lane_addr = uint32_t(quarter * 32) << 16;
    const int c0 = half * 32;                               // this thread's 32 of the 64 channels
    const float a2 = -expf(to_f(p.a_log[h])) * 1.4426950408889634f;
    const float dk = to_f(p.dskip[h]);
    const int pn = min(SC_PB, p.P - p0);
    const float* dt = p.dt + (size_t)h * p.b.T + row0;
    float* gs = p.state + (((size_t)p.b.row[seq] * p.H + h) * p.N + t) * p.P + p0 + c0;
    const size_t seg_i = p.seg_chunks > 0 ? ((size_t)seq * p.H + h) * p.n_seg + seg : 0;
    float* ss = p.seg_state + (seg_i * p.N + t) * p.P + p0 + c0;
    float log2_sum = 0.f;
    uint32_t r[32];
    {
      const bool segs = p.seg_chunks > 0;
      const bool have = !STATE_ONLY && t < p.N && (segs || p.b.start[seq] != 0);
      const float* from = segs ? ss : gs;
#pragma unroll
      for (int j = 0; j < 32; ++j) r[j] = (have && c0 + j < pn) ? __float_as_uint(from[j]) : 0u;
      tmem_st_32x32b_x16(tm_s + lane_addr + c0, r);
      tmem_st_32x32b_x16(tm_s + lane_addr + c0 + 16, r + 16);
      tmem_st_wait();
    }
    float dt_next = t < len ? dt[t] : 0.f;
    // after a wait that ran out the thread keeps step with the named barriers and stores nothing
    bool ok = true;
    for (int c = 0; c < n_chunks; ++c) {
      const uint32_t ph = c & 1;
      const int tok = c * SC_Q + t;
      // ---- step sizes and the running sum of log2 decays
      const float dtv = dt_next;
      dt_next = tok + SC_Q < len ? dt[tok + SC_Q] : 0.f;
      // sums inside the row's block of 32 tokens, from its start up to t and behind t to its end (scanned both ways: a
      // difference of prefix sums would lose the small distances behind a stretch of fast decay)
      float pre = a2 * dtv, suf = pre;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float u = __shfl_up_sync(0xffffffffu, pre, o), v = __shfl_down_sync(0xffffffffu, suf, o);
        if (lane >= o) pre += u;
        if (lane + o < 32) suf += v;
      }
      suf = __shfl_down_sync(0xffffffffu, suf, 1);
      if (lane == 31) suf = 0.f;
      if (half == 0 && lane == 31) wtot[quarter] = pre;
      asm volatile("bar.sync 1, 256;" ::: "memory");
      const float b0 = wtot[0], b1 = wtot[1], b2 = wtot[2], b3 = wtot[3];
      // from the end of block q (0, 1, 2) to this row's block, and from there to the end of the chunk
      const float gap2 = 0.f, gap1 = quarter > 2 ? b2 : 0.f, gap0 = quarter > 2 ? b1 + b2 : quarter > 1 ? b1 : 0.f;
      const float ahead = quarter == 0 ? b1 + b2 + b3 : quarter == 1 ? b2 + b3 : quarter == 2 ? b3 : 0.f;
      const float cum = pre + (quarter == 0 ? 0.f : b0 + gap0), total = b0 + b1 + b2 + b3;
      log2_sum += total;
      // a block of 32 tokens in front of this row's weighs its token s with e^{sum behind s} dt_s, the same for all rows,
      // and the row adds the decay from the block's end to itself
      if (half == 0) wsm[t] = ex2(suf) * dtv;
      const float w_own = pre - lg2(dtv);                   // for the diagonal block; dt = 0: +inf, the weight vanishes
      // ---- S: bf16 hi / lo rows for the read-out, decayed in place for the update
      tmem_ld_32x32b_x32(tm_s + lane_addr + c0, r);
      tmem_ld_wait();
      {
        const float decay = ex2(total);
        uint8_t* s_hi = smem + ScSmem::S_OFF;
        uint8_t* s_lo = s_hi + 16384;
        if (!STATE_ONLY) {
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int u = 0; u < 4; ++u)
              split2(__uint_as_float(r[8 * j + 2 * u]), __uint_as_float(r[8 * j + 2 * u + 1]), hi[u], lo[u]);
            const int off = sw128(t, half * 4 + j);
            *reinterpret_cast<uint4*>(s_hi + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
            *reinterpret_cast<uint4*>(s_lo + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
          }
        }
#pragma unroll
        for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * decay);
        tmem_st_32x32b_x16(tm_s + lane_addr + c0, r);
        tmem_st_32x32b_x16(tm_s + lane_addr + c0 + 16, r + 16);
        tmem_st_wait();
        fence_proxy_async_smem();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(s_ready);
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");        // wsm is complete
      if (!STATE_ONLY) {
        ok = ok &&   mbar_wait(g_full, ph, p.status, ERR_TIMEOUT_TMEM_FULL);
        tc_fence_after();
      }
      // ---- weighted scores of the 32-column blocks half and half + 2 (blocks behind the diagonal are zero); all of G
      //      is read before M overwrites it
      if (!STATE_ONLY) {
        uint32_t m_hi[2][16], m_lo[2][16];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int q = half + 2 * u;
          if (q < quarter) {
            tmem_ld_32x32b_x32(tm_g + lane_addr + q * 32, r);
            const float rs = ex2(pre + (q == 0 ? gap0 : q == 1 ? gap1 : gap2));
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 32; j += 4) {
              const float4 w = *reinterpret_cast<const float4*>(wsm + q * 32 + j);
              split2(w.x * rs * __uint_as_float(r[j]), w.y * rs * __uint_as_float(r[j + 1]), m_hi[u][j / 2], m_lo[u][j / 2]);
              split2(w.z * rs * __uint_as_float(r[j + 2]), w.w * rs * __uint_as_float(r[j + 3]), m_hi[u][j / 2 + 1], m_lo[u][j / 2 + 1]);
            }
          } else if (q == quarter) {
            tmem_ld_32x32b_x32(tm_g + lane_addr + q * 32, r);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 32; j += 2) {
              const float w0 = __shfl_sync(0xffffffffu, w_own, j), w1 = __shfl_sync(0xffffffffu, w_own, j + 1);
              const float a = j <= lane ? ex2(pre - w0) * __uint_as_float(r[j]) : 0.f;
              const float b = j + 1 <= lane ? ex2(pre - w1) * __uint_as_float(r[j + 1]) : 0.f;
              split2(a, b, m_hi[u][j / 2], m_lo[u][j / 2]);
            }
          } else {
#pragma unroll
            for (int j = 0; j < 16; ++j) { m_hi[u][j] = 0u; m_lo[u][j] = 0u; }
          }
        }
        tc_fence_before();
        asm volatile("bar.sync 1, 256;" ::: "memory");
        tc_fence_after();
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          const int q = half + 2 * u;
          tmem_st_32x32b_x16(tm_g + lane_addr + q * 16, m_hi[u]);
          tmem_st_32x32b_x16(tm_g + lane_addr + 64 + q * 16, m_lo[u]);
        }
        const float e = ex2(cum);
        tmem_ld_32x32b_x32(tm_y + lane_addr + c0, r);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * e);
        tmem_st_32x32b_x16(tm_y + lane_addr + c0, r);
        tmem_st_32x32b_x16(tm_y + lane_addr + c0 + 16, r + 16);
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(m_ready);
      }
      // ---- weighted inputs into the S tiles (their MMAs are complete); x stays in registers for the skip term
      uint4 x[4];
      {
        const float w = ex2(suf + ahead) * dtv;
        ok = ok && mbar_wait(x_full, ph, p.status, ERR_TIMEOUT_FULL);
        const uint8_t* xs = smem + ScSmem::X_OFF;
        uint8_t* w_hi = smem + ScSmem::S_OFF;
        uint8_t* w_lo = w_hi + 16384;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int off = sw128(t, half * 4 + j);
          x[j] = *reinterpret_cast<const uint4*>(xs + off);
          const __nv_bfloat162* x2 = reinterpret_cast<const __nv_bfloat162*>(&x[j]);
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            const float2 f = __bfloat1622float2(x2[u]);
            split2(f.x * w, f.y * w, hi[u], lo[u]);
          }
          *reinterpret_cast<uint4*>(w_hi + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(w_lo + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
        fence_proxy_async_smem();
        __syncwarp();
        if (lane == 0) mbar_arrive(xw_ready);
      }
      ok = ok && mbar_wait(done, ph, p.status, ERR_TIMEOUT_TMEM_FULL);
      tc_fence_after();
      if (STATE_ONLY) continue;
      // ---- y = Y + D x
      tmem_ld_32x32b_x32(tm_y + lane_addr + c0, r);
      tmem_ld_wait();
      // staged in the x tile so that the rows leave in whole lines
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const __nv_bfloat162* x2 = reinterpret_cast<const __nv_bfloat162*>(&x[j]);
        uint32_t w[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float2 f = __bfloat1622float2(x2[u]);
          w[u] = pack_bf16x2(fmaf(dk, f.x, __uint_as_float(r[8 * j + 2 * u])), fmaf(dk, f.y, __uint_as_float(r[8 * j + 2 * u + 1])));
        }
        *reinterpret_cast<uint4*>(smem + ScSmem::X_OFF + sw128(t, half * 4 + j)) = make_uint4(w[0], w[1], w[2], w[3]);
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");
      const int rows = min(SC_Q, len - c * SC_Q);
      __nv_bfloat16* yc = p.y + (size_t)(row0 + c * SC_Q) * p.inner + h * p.P + p0;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int rr = i * 32 + (threadIdx.x >> 3), j = threadIdx.x & 7;
        const uint4 v = *reinterpret_cast<const uint4*>(smem + ScSmem::X_OFF + sw128(rr, j));
        if (ok && rr < rows && j * 8 < pn) *reinterpret_cast<uint4*>(yc + (size_t)rr * p.inner + j * 8) = v;
      }
    }
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      tmem_ld_32x32b_x32(tm_s + lane_addr + c0, r);         // all lanes take part
      tmem_ld_wait();
      float* to = STATE_ONLY ? ss : gs;
      if (t < p.N && (STATE_ONLY || (last && p.b.live(seq)))) {
#pragma unroll
        for (int j = 0; j < 32; j += 4)
          if (c0 + j < pn) *reinterpret_cast<uint4*>(to + j) = make_uint4(r[j], r[j + 1], r[j + 2], r[j + 3]);
      }
      if (STATE_ONLY && threadIdx.x == 0 && p0 == 0) p.seg_log2[seg_i] = log2_sum;
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
  if (warp == 8) {
    tc_fence_after();
    tmem_dealloc(tmem, 256);
  }
}

// Between the passes: every segment's contribution becomes the state at its start.
__global__ void __launch_bounds__(256)
ssd_segment_kernel(const SsdChunkParams p) {
  const int h = blockIdx.x, seq = blockIdx.y, np = p.N * p.P;
  const int len = p.b.cu[seq + 1] - p.b.cu[seq];
  const int segs = (len + p.seg_chunks * SC_Q - 1) / (p.seg_chunks * SC_Q);
  const size_t s0 = ((size_t)seq * p.H + h) * p.n_seg;
  const float* gs = p.state + ((size_t)p.b.row[seq] * p.H + h) * np;
  const bool fresh = p.b.start[seq] == 0;
  for (int i = blockIdx.z * 256 + threadIdx.x; i < np; i += gridDim.z * 256) {
    float v = fresh ? 0.f : gs[i];
    for (int g = 0; g < segs; ++g) {
      float* q = p.seg_state + (s0 + g) * np + i;
      const float own = g + 1 < segs ? *q : 0.f;
      *q = v;
      if (g + 1 < segs) v = fmaf(ex2(p.seg_log2[s0 + g]), v, own);
    }
  }
}

}  // namespace b200

using namespace b200;

// Whether the kernel covers these sizes: TMA column starts and 16-byte rows, whole K steps of the contraction over N.
extern "C" int b200_ssd_chunk_fits(int H, int P, int N, int G) {
  const int inner = H * P, cc = inner + 2 * G * N;
  return cc % 8 == 0 && P % 8 == 0 && inner % 8 == 0 && N % 16 == 0 && N <= 128 ? 1 : 0;
}

// bf16 scan of a ragged batch; like b200_ssd_scan with f32 = 0. seg_chunks > 0: portions are cut into n_seg
// segments of that many chunks (n_seg * seg_chunks * 128 tokens cover the longest); seg_state holds n * H * n_seg * N * P
// floats, seg_log2 n * H * n_seg.
extern "C" int b200_ssd_chunk(const void* xbc, const float* dt, const int* cu, const int* start, const int* row,
                              const int* active, const int* tok_seq, int n, int T, const void* a_log, const void* dskip,
                              float* state, void* y, int H, int P, int N, int G, int seg_chunks, int n_seg,
                              float* seg_state, float* seg_log2, int* status, void* stream) {
  if (T <= 0 || n <= 0) return 0;
  if (seg_chunks > 0 && (n_seg < 1 || seg_state == nullptr || seg_log2 == nullptr ||
                         (reinterpret_cast<uintptr_t>(seg_state) & 15))) return -11;
  if (H % G || n > 65535 || !b200_ssd_chunk_fits(H, P, N, G)) return -10;
  if ((reinterpret_cast<uintptr_t>(xbc) | reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(state)) & 15) return -12;
  const int inner = H * P, cc = inner + 2 * G * N;
  CUtensorMap tm;
  if (int r = make_tmap_bf16_2d(&tm, xbc, T, cc, cc, SC_Q, 64)) return r;
  static std::atomic<unsigned long long> c0{0}, c1{0};
  if (!set_max_smem_once(c0, ssd_chunk_kernel<false>, ScSmem::TOTAL)) return -2;
  if (!set_max_smem_once(c1, ssd_chunk_kernel<true>, ScSmem::TOTAL)) return -2;
  SsdChunkParams p;
  p.dt = dt; p.a_log = reinterpret_cast<const __nv_bfloat16*>(a_log); p.dskip = reinterpret_cast<const __nv_bfloat16*>(dskip);
  p.state = state; p.y = reinterpret_cast<__nv_bfloat16*>(y); p.b = make_ragged(cu, start, row, active, tok_seq, n, T);
  p.H = H; p.P = P; p.N = N; p.G = G; p.inner = inner; p.status = status;
  p.pblocks = (P + SC_PB - 1) / SC_PB;
  p.seg_chunks = seg_chunks > 0 ? seg_chunks : 0; p.n_seg = seg_chunks > 0 ? n_seg : 1;
  p.seg_state = seg_state; p.seg_log2 = seg_log2;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid(H, n, p.pblocks * p.n_seg);
  if (p.seg_chunks > 0) {
    ssd_chunk_kernel<true><<<grid, 288, ScSmem::TOTAL, st>>>(tm, p);
    ssd_segment_kernel<<<dim3(H, n, (N * P + 255) / 256), 256, 0, st>>>(p);
  }
  ssd_chunk_kernel<false><<<grid, 288, ScSmem::TOTAL, st>>>(tm, p);
  return cudaGetLastError() == cudaSuccess ? 0 : -3;
}
