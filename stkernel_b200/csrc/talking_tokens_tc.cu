// Talking-heads attention of decode rows and short spans on the 5th-generation tensor cores (bf16): mixed queries against the keys of all
// key/value heads side by side, then every head sums the values of its own key/value head.
//
// One CTA per (split of the key range, tile of tokens, group of heads).  The tile's (token, head) pairs are N = 16 or 32 columns:
//
//   loader warp      per block of 128 rows (two pages) by TMA: the key columns as pairs of 64-column panels, then the value columns, all
//                    through one ring in the order in which they are used (the keys of the next block come before the values)
//   MMA warp         S^T[key, column] = keys . Q^T as the panels arrive, one block ahead of the softmax; O^T[dim, column] += values^T . P
//                    with the value panels as MN-major operand, 128 dims at a time
//   softmax warps    eight, one key and half of the columns per thread: column maxima over the lanes, probabilities to shared memory as
//                    bf16 pairs (high parts and remainders are 2N columns of one product), O rescaled only when a column's maximum
//                    grew by more than 2^8
//
// Of O^T[dim, column] the dims of the column's own key/value head are kept.  Each CTA writes an unnormalised partial result;
// talking_merge joins the splits, counts the sink and applies the gate.  Value rows outside the visible keys are zeroed in shared
// memory, so what an earlier owner left in a page cannot reach a sum (scores there are replaced).  Every mbarrier wait is bounded.
#define STK_PDL_CLASS 128
#include "latent_attention.cuh"
#include "talking_attention.cuh"
#include "warp_reduce.cuh"

namespace stk {

int make_tmap_2d(CUtensorMap* tm, const void* base, int elem_bytes, long long rows, long long cols, long long ld, int box_rows);

constexpr int kTtBlock = 128, kTtPanel = kTtBlock * 128, kTtThreads = 320, kTtMaxPairs = 6, kTtMaxSplits = 64;
constexpr float kTtLog2e = 1.4426950408889634f;

struct TtArgs {
  TalkArgs a;
  const int* query_start; const int* req_rows; const int* start_pos;
  int n_req, max_span;
  int tq, hs;                            // tokens per tile, heads per group (tq * hs <= N)
  int k_pairs, slots;                    // panel pairs of a row's keys, ring size
  float* part;                           // [splits][T][H][V + 2]
  int T;
  int* status;
};

struct alignas(8) TtBars {
  uint64_t full[kTtMaxPairs], empty[kTtMaxPairs];
  uint64_t s_full[2], p_full, pv_done, clean;
  uint32_t tmem_base;
  int find[2];
};

__device__ __forceinline__ float tt_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Barrier of the softmax warps that also tells whether every one of them is fine: they leave their loop together.
__device__ __forceinline__ bool tt_bar_all(bool ok) {
  int r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.s32 p, %1, 0;\n\t"
      "barrier.cta.red.and.pred q, 1, 256, p;\n\t"
      "selp.s32 %0, 1, 0, q;\n\t}"
      : "=r"(r) : "r"(ok ? 1 : 0) : "memory");
  return r != 0;
}
__device__ __forceinline__ void tt_bar_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
__device__ __forceinline__ void tt_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
      "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
// 8 or 16 columns of the warp's 32 lanes
template <int C>
__device__ __forceinline__ void tt_ld(uint32_t taddr, uint32_t (&r)[C]) {
  if constexpr (C == 16) {
    tmem_ld_32x16(taddr, r);
  } else {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                 : "r"(taddr));
  }
}

template <int N>
__global__ void __launch_bounds__(kTtThreads, 1)
talking_tokens_tc_kernel(const __grid_constant__ CUtensorMap tm_rows, const TtArgs x) {
  extern __shared__ uint8_t smem_raw[];
  const TalkArgs& a = x.a;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int KD = a.G * a.kp, q_panels = 2 * x.k_pairs;
  uint8_t* ring = smem;                                             // [slots][2 panels][128 rows x 128 B]
  uint8_t* q_s = ring + x.slots * 2 * kTtPanel;                     // [q_panels][N x 128 B]
  uint8_t* p_s = q_s + q_panels * N * 128;                          // [2 key panels][2N x 128 B]: high parts, remainders
  TtBars* bars = reinterpret_cast<TtBars*>(p_s + 2 * 2 * N * 128);
  float* smax = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(bars) + 256);   // [4][N]
  float* m_ref = smax + 4 * N;                                      // [N]
  float* alpha = m_ref + N;                                         // [N]
  int* col_pos = reinterpret_cast<int*>(alpha + N);                 // [N] last key a column sees (-1: padding)
  int* col_lo = col_pos + N;                                        // [N] first key a column sees
  int* col_row = col_lo + N;                                        // [N] token * heads + head of a column
  int* col_v = col_row + N;                                         // [N] first value dim of the column's key/value head
  int* flags = col_v + N;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_trigger();
  if (warp == 0) {
    // the tile's request: 32 requests at a time
    int left = blockIdx.y, ri = -1, off = 0;
    for (int i0 = 0; i0 < x.n_req && ri < 0; i0 += 32) {
      const int i = i0 + lane;
      int tiles = 0;
      if (i < x.n_req) {
        const int n = x.query_start[i + 1] - x.query_start[i];
        if (n > 0 && n <= x.max_span) tiles = (n + x.tq - 1) / x.tq;
      }
      int incl = tiles;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += v;
      }
      const unsigned hit = __ballot_sync(0xffffffffu, left < incl);
      if (hit) {
        const int src = __ffs(hit) - 1;
        ri = i0 + src;
        off = left - (__shfl_sync(0xffffffffu, incl, src) - __shfl_sync(0xffffffffu, tiles, src));
      } else {
        left -= __shfl_sync(0xffffffffu, incl, 31);
      }
    }
    if (lane == 0) {
      bars->find[0] = ri;
      bars->find[1] = off * x.tq;
    }
  } else if (threadIdx.x == 288) {
    for (int s = 0; s < kTtMaxPairs; ++s) {
      mbar_init(&bars->full[s], 1);
      mbar_init(&bars->empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) mbar_init(&bars->s_full[i], 1);
    mbar_init(&bars->p_full, 8);
    mbar_init(&bars->pv_done, 1);
    mbar_init(&bars->clean, 1);
    fence_barrier_init();
  }
  __syncthreads();
  const int ri = bars->find[0];
  if (ri < 0) return;
  const int off = bars->find[1];
  const int h0 = blockIdx.z * x.hs, nh = min(x.hs, a.H - h0);
  // 128-dim tiles of the values of the group's key/value heads
  const int v0 = h0 / (a.H / a.G) * a.vp / kTtBlock, v_tiles = ((h0 + nh - 1) / (a.H / a.G) * a.vp + a.vp - 1) / kTtBlock + 1 - v0;
  const int tok0 = x.query_start[ri] + off, ntok = min(x.tq, x.query_start[ri + 1] - tok0);
  const int p0 = x.start_pos[ri] + off, p_last = p0 + ntok - 1;
  const int k_first = talk_first(a, p0), first_b = k_first / kTtBlock, end_b = p_last / kTtBlock + 1, blocks = end_b - first_b;
  const int per = (blocks + gridDim.x - 1) / gridDim.x;
  const int b0 = first_b + min(blocks, static_cast<int>(blockIdx.x) * per), b1 = min(end_b, b0 + per);
  float* part = x.part + static_cast<long long>(blockIdx.x) * x.T * a.H * (a.V + 2);
  if (b0 >= b1) {
    for (int e = threadIdx.x; e < ntok * nh; e += kTtThreads) {
      float* o = part + (static_cast<long long>(tok0 + e / nh) * a.H + h0 + e % nh) * (a.V + 2);
      o[a.V] = -INFINITY;
      o[a.V + 1] = 0.f;
    }
    return;
  }
  const int* bt = a.table + static_cast<long long>(x.req_rows[ri]) * a.bt_stride;
  auto page_of = [&](int lp) { return lp <= p_last / kTkPage ? max(bt[lp], 0) : 0; };
  auto load_pair = [&](int st, int col, int pg0, int pg1) {
    mbar_expect_tx(&bars->full[st], 2 * kTtPanel);
    uint8_t* dst = ring + st * 2 * kTtPanel;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      tma_load_2d(dst + j * kTtPanel, &tm_rows, &bars->full[st], col + j * 64, pg0 * kTkPage);
      tma_load_2d(dst + j * kTtPanel + kTtPanel / 2, &tm_rows, &bars->full[st], col + j * 64, pg1 * kTkPage);
    }
  };
  // the first block's keys are on their way while the queries are laid out
  const int early = min(x.k_pairs, x.slots);
  if (warp == 8 && lane == 0) {
    const int pg0 = page_of(2 * b0), pg1 = page_of(2 * b0 + 1);
    for (int d = 0; d < early; ++d) load_pair(d, a.k_col + d * 128, pg0, pg1);
  }
  if (warp == 9) {
    tmem_alloc(&bars->tmem_base, 512);
    tmem_relinquish();
  }
  __syncwarp();
  // the queries, in the layout of the products' operand
  for (int n = warp; n < N; n += kTtThreads / 32) {
    const int q = n / x.hs, hh = n - q * x.hs;
    const bool valid = q < ntok && hh < nh;
    const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(a.q) + (valid ? (static_cast<long long>(h0 + hh) * x.T + tok0 + q) * KD : 0);
    for (int cc = lane; cc < q_panels * 8; cc += 32) {
      uint4 v = make_uint4(0, 0, 0, 0);
      if (valid && cc * 8 < KD) v = *reinterpret_cast<const uint4*>(src + cc * 8);
      *reinterpret_cast<uint4*>(q_s + (cc >> 3) * (N * 128) + n * 128 + (((cc & 7) ^ (n & 7)) << 4)) = v;
    }
    if (lane == 0) {
      col_pos[n] = valid ? p0 + q : -1;
      col_lo[n] = talk_first(a, p0 + q);
      col_row[n] = (tok0 + q) * a.H + h0 + hh;
      col_v[n] = (h0 + hh) / (a.H / a.G) * a.vp;
      m_ref[n] = -INFINITY;
    }
  }
  if (threadIdx.x < 2) flags[threadIdx.x] = 0;
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_base;                            // scores: two buffers of N columns; outputs from column 2N on
  const uint32_t tmem_o = tmem + 2 * N;
  // rows of a block that no token of the tile sees: before the first key, behind the last one
  const int front = max(0, k_first - b0 * kTtBlock);
  const int back = b1 == end_b ? (p_last + 1) % kTtBlock : 0;       // 0: none
  auto dirty = [&](int b) { return (b == b0 && front > 0) || (b == b1 - 1 && back > 0); };

  if (warp == 8) {
    // ------------------------------- loader -------------------------------
    bool ok = true;
    int seq = early;
    auto load = [&](int col, int pg0, int pg1) {                    // one pair, lane 0
      const int st = seq % x.slots;
      if (seq >= x.slots) ok = mbar_wait(&bars->empty[st], ((seq / x.slots) - 1) & 1, x.status, 930);
      if (ok) {
        load_pair(st, col, pg0, pg1);
        ++seq;
      }
    };
    auto load_keys = [&](int b, int done) {
      const int pg0 = page_of(2 * b), pg1 = page_of(2 * b + 1);
      for (int d = done; d < x.k_pairs && ok; ++d) load(a.k_col + d * 128, pg0, pg1);
    };
    if (lane == 0) load_keys(b0, early);
    for (int b = b0; b < b1; ++b) {
      if (lane == 0) {
        if (ok && b + 1 < b1) load_keys(b + 1, 0);
        const int pg0 = page_of(2 * b), pg1 = page_of(2 * b + 1);
        for (int j = 0; j < v_tiles && ok; ++j) load((v0 + j) * 128, pg0, pg1);
      }
      ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
      if (!ok) break;
      if (dirty(b)) {
        const int last = __shfl_sync(0xffffffffu, seq, 0);
        const int r0 = b == b0 ? front : 0, r1 = b == b1 - 1 && back > 0 ? back : kTtBlock;
        for (int s = last - v_tiles; s < last && ok; ++s) {
          const int st = s % x.slots;
          ok = mbar_wait(&bars->full[st], (s / x.slots) & 1, x.status, 931);
          ok = __all_sync(0xffffffffu, ok);
          for (int e = lane; e < 2 * kTtBlock * 8; e += 32) {
            const int row = (e >> 3) & (kTtBlock - 1);
            if (row < r0 || row >= r1) *reinterpret_cast<uint4*>(ring + st * 2 * kTtPanel + e * 16) = make_uint4(0, 0, 0, 0);
          }
        }
        fence_proxy_async();
        __syncwarp();
        if (ok && lane == 0) mbar_arrive(&bars->clean);
        if (!ok) break;
      }
    }
    if (!ok && lane == 0) {
      // leave no copy in flight: what was asked for lands before the CTA's shared memory goes away
      for (int s = max(0, seq - x.slots); s < seq; ++s) mbar_wait(&bars->full[s % x.slots], (s / x.slots) & 1, nullptr, 0);
    }
    __syncwarp();
  } else if (warp == 9) {
    // ------------------------------- MMA issuer -------------------------------
    constexpr uint32_t kIdescS = umma_idesc(1u, 1u, 128, N);
    constexpr uint32_t kIdescO = umma_idesc(1u, 1u, 128, 2 * N) | (1u << 15);             // A is MN-major
    constexpr uint32_t kStep = kTtPanel >> 4, kQStep = (N * 128) >> 4;                    // panels in descriptor units
    const uint32_t lead = elect_one() ? 1u : 0u, tm = __shfl_sync(0xffffffffu, tmem, 0);
    const uint32_t k_lo = desc_lo(smem_u32(ring)), v_lo = desc_lo(smem_u32(ring), kTtPanel);
    const uint32_t q_lo = desc_lo(smem_u32(q_s)), p_lo = desc_lo(smem_u32(p_s));
    int slot = 0;
    uint32_t par = 0u, cleaned = 0u;
    auto next = [&]() {
      if (++slot == x.slots) { slot = 0; par ^= 1u; }
    };
    auto scores = [&](int b) {
      const uint32_t d0 = tm + ((b - b0) & 1) * N;
      for (int d = 0; d < x.k_pairs; ++d) {
        if (!mbar_wait(&bars->full[slot], par, x.status, 932)) return false;
        tc_fence_after();
        const uint32_t al = k_lo + slot * 2 * kStep, bl = q_lo + d * 2 * kQStep;
#pragma unroll
        for (int ks = 0; ks < 8; ++ks)
          mma_ss(d0, al + (ks >> 2) * kStep + 2 * (ks & 3), bl + (ks >> 2) * kQStep + 2 * (ks & 3), kIdescS,
                 ks > 0 ? 1u : (d > 0 ? 1u : 0u), lead);
        mma_commit(&bars->empty[slot], lead);
        next();
      }
      mma_commit(&bars->s_full[(b - b0) & 1], lead);
      return true;
    };
    bool ok = scores(b0);
    for (int b = b0; b < b1 && ok; ++b) {
      const int i = b - b0;
      if (b + 1 < b1) ok = scores(b + 1);
      if (ok) ok = mbar_wait(&bars->p_full, i & 1, x.status, 933);
      if (ok && dirty(b)) {
        ok = mbar_wait(&bars->clean, cleaned, x.status, 934);
        cleaned ^= 1u;
      }
      if (!ok) break;
      tc_fence_after();
      for (int j = 0; j < v_tiles; ++j) {
        if (!mbar_wait(&bars->full[slot], par, x.status, 935)) { ok = false; break; }
        tc_fence_after();
        const uint32_t al = v_lo + slot * 2 * kStep, dj = tm + 2 * N + j * 2 * N;
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          mma_ss(dj, al + kk * 128, p_lo + (kk >> 2) * 2 * kQStep + 2 * (kk & 3), kIdescO, kk > 0 ? 1u : (i > 0 ? 1u : 0u), lead);
        mma_commit(&bars->empty[slot], lead);
        next();
      }
      if (ok) mma_commit(&bars->pv_done, lead);
    }
    __syncwarp();
  } else {
    // ------------------------------- softmax -------------------------------
    constexpr int NH = N / 2;                                       // columns of this thread
    const int row = (warp & 3) * 32 + lane, c0 = (warp >> 2) * NH;
    const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const float c_in = a.scale * kTtLog2e;
    float l[NH];
#pragma unroll
    for (int n = 0; n < NH; ++n) l[n] = 0.f;
    bool ok = true;
    for (int b = b0; b < b1; ++b) {
      const int i = b - b0, key = b * kTtBlock + row;
      ok = ok && mbar_wait(&bars->s_full[i & 1], (i >> 1) & 1, x.status, 936);
      tc_fence_after();
      float v[NH], keep[NH];
      {
        uint32_t r[NH];
        tt_ld<NH>(tmem + (i & 1) * N + c0 + lanes, r);
        tmem_ld_wait();
#pragma unroll
        for (int n = 0; n < NH; ++n) {
          v[n] = __uint_as_float(r[n]) * c_in;
          if (key > col_pos[c0 + n] || key < col_lo[c0 + n]) v[n] = -INFINITY;
        }
      }
#pragma unroll
      for (int n = 0; n < NH; ++n) keep[n] = v[n];
      bfly_reduce_store<NH, true>(v, smax + (warp & 3) * N + c0, lane);
      ok = tt_bar_all(ok);
      if (!ok) break;
      if (threadIdx.x == 0) flags[(i + 1) & 1] = 0;
      if (threadIdx.x < N) {
        const int n = threadIdx.x;
        const float bm = fmaxf(fmaxf(smax[n], smax[N + n]), fmaxf(smax[2 * N + n], smax[3 * N + n]));
        const float mo = m_ref[n];
        float f = 1.f;
        if (bm > mo + 8.f || (mo == -INFINITY && bm > -INFINITY)) {
          f = mo == -INFINITY ? 0.f : tt_ex2(mo - bm);
          m_ref[n] = bm;
          flags[i & 1] = 1;
        }
        alpha[n] = f;
      }
      tt_bar_sync();
      if (i > 0) {
        // the previous product has read the probabilities and finished its output
        ok = mbar_wait(&bars->pv_done, (i - 1) & 1, x.status, 937);
        if (!ok) continue;
        tc_fence_after();
      }
      if (flags[i & 1]) {
#pragma unroll
        for (int n = 0; n < NH; ++n) l[n] *= alpha[c0 + n];
        if (i > 0) {
          // high parts for the first four warps, remainders for the others
          const uint32_t to = tmem_o + (warp >> 2) * N + lanes;
          for (int j = 0; j < v_tiles; ++j)
#pragma unroll
            for (int c = 0; c < N; c += 16) {
              uint32_t o[16];
              tmem_ld_32x16(to + j * 2 * N + c, o);
              tmem_ld_wait();
#pragma unroll
              for (int k = 0; k < 16; ++k) o[k] = __float_as_uint(__uint_as_float(o[k]) * alpha[c + k]);
              tt_st16(to + j * 2 * N + c, o);
            }
          asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        }
      }
      uint8_t* dst = p_s + (row >> 6) * (2 * N * 128) + c0 * 128 + (row & 7) * 2;
      const int chunk = (row & 63) >> 3;
#pragma unroll
      for (int n = 0; n < NH; ++n) {
        const float mr = m_ref[c0 + n];
        const float p = mr == -INFINITY ? 0.f : tt_ex2(keep[n] - mr);
        l[n] += p;
        const __nv_bfloat16 hi = __float2bfloat16(p);
        const int at = n * 128 + ((chunk ^ (n & 7)) << 4);
        *reinterpret_cast<__nv_bfloat16*>(dst + at) = hi;
        *reinterpret_cast<__nv_bfloat16*>(dst + N * 128 + at) = __float2bfloat16(p - bf16_to_f(hi));
      }
      fence_proxy_async();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->p_full);
    }
    if (ok) ok = mbar_wait(&bars->pv_done, (b1 - 1 - b0) & 1, x.status, 938);
    tc_fence_after();
    bfly_reduce_store<NH, false>(l, smax + (warp & 3) * N + c0, lane);
    tt_bar_sync();
    if (ok) {
      // the two halves of the warps take every other 128 dims
      for (int j = warp >> 2; j < v_tiles; j += 2) {
        const int d = (v0 + j) * 128 + row;
#pragma unroll
        for (int c = 0; c < N; c += 16) {
          uint32_t u[16], w[16];
          tmem_ld_32x16(tmem_o + j * 2 * N + c + lanes, u);
          tmem_ld_32x16(tmem_o + j * 2 * N + N + c + lanes, w);
          tmem_ld_wait();
#pragma unroll
          for (int k = 0; k < 16; ++k) {
            const int vd = d - col_v[c + k];
            if (col_pos[c + k] >= 0 && vd >= 0 && vd < a.V)
              part[static_cast<long long>(col_row[c + k]) * (a.V + 2) + vd] = __uint_as_float(u[k]) + __uint_as_float(w[k]);
          }
        }
      }
      if (threadIdx.x < N && col_pos[threadIdx.x] >= 0) {
        const int n = threadIdx.x;
        float* o = part + static_cast<long long>(col_row[n]) * (a.V + 2);
        o[a.V] = m_ref[n];
        o[a.V + 1] = (smax[n] + smax[N + n]) + (smax[2 * N + n] + smax[3 * N + n]);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// One CTA per (token, head): joins the splits, counts the sink, normalises, gates; zeros for padding tokens and behind the last head.
__global__ void __launch_bounds__(128)
talking_merge_kernel(const TalkArgs a, const float* __restrict__ part, int splits, const int* __restrict__ first_pos,
                     const int* __restrict__ last_pos, int max_span, int T) {
  __shared__ float wt[kTtMaxSplits];
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const int h = blockIdx.y;
  const bool live = a.tok_req[t] >= 0 && a.positions[t] >= 0;
  if (live && last_pos[t] - first_pos[t] + 1 > max_span) return;
  __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(a.out) + t * a.ldo;
  if (h == a.H - 1)
    for (int d = a.H * a.V + threadIdx.x; d < a.out_cols; d += blockDim.x) o[d] = __float2bfloat16(0.f);
  o += h * a.V;
  if (!live) {
    for (int d = threadIdx.x; d < a.V; d += blockDim.x) o[d] = __float2bfloat16(0.f);
    return;
  }
  const long long step = static_cast<long long>(T) * a.H * (a.V + 2);
  const float* p = part + (t * a.H + h) * (a.V + 2);
  if (threadIdx.x < 32) {
    // the splits' weights: two per lane; maxima are in units of log2(e)
    float m[2], l[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = threadIdx.x + i * 32;
      m[i] = s < splits ? p[s * step + a.V] : -INFINITY;
      l[i] = s < splits ? p[s * step + a.V + 1] : 0.f;
    }
    const float sink = a.sink != nullptr ? a.sink[h] * kTtLog2e : -INFINITY;
    const float mx = fmaxf(warp_max(fmaxf(m[0], m[1])), sink);
    float sum = 0.f, f[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      f[i] = m[i] == -INFINITY ? 0.f : tt_ex2(m[i] - mx);
      sum = fmaf(f[i], l[i], sum);
    }
    sum = warp_sum(sum);
    if (a.sink != nullptr) sum += tt_ex2(sink - mx);
    const float g = talk_gate(a, t, h) / sum;
    wt[threadIdx.x] = f[0] * g;
    wt[threadIdx.x + 32] = f[1] * g;
  }
  __syncthreads();
  for (int d = threadIdx.x; d < a.V; d += blockDim.x) {
    float v = 0.f;
    // a split without keys left its columns unwritten
#pragma unroll 4
    for (int s = 0; s < splits; ++s) {
      const float w = wt[s];
      v = fmaf(w, w != 0.f ? p[s * step + d] : 0.f, v);
    }
    o[d] = __float2bfloat16(v);
  }
}

struct TtShape { int n, hs, k_pairs, v_tiles, slots; };
static int tt_fixed(const TtShape& s) { return 2 * s.k_pairs * s.n * 128 + 4 * s.n * 128 + 256 + 10 * s.n * 4 + 64 + 1024; }
// Groups of `hs` heads; 0: as many as fit.  n 0: the kernel does not cover the layer.
static TtShape tt_shape(int H, int G, int kp, int vp, int max_span, int hs = 0) {
  TtShape s = {};
  s.k_pairs = (G * kp + 127) / 128;
  s.v_tiles = (G * vp + 127) / 128;
  const bool wide = hs > 0 ? hs > 16 : H > 16 || (max_span > 1 && 2 * H > 16);
  for (int n = wide ? 32 : 16; n >= 16 && hs <= n; n -= 16) {
    s.n = n;
    const int groups = (H + n - 1) / n;
    s.hs = hs > 0 ? hs : (H + groups - 1) / groups;
    s.slots = (227 * 1024 - tt_fixed(s)) / (2 * kTtPanel);
    if (s.slots > kTtMaxPairs) s.slots = kTtMaxPairs;
    // the values of a block lie in the ring while rows that nobody sees are zeroed
    if (s.slots >= s.v_tiles && s.slots >= 3 && (2 + 2 * s.v_tiles) * n <= 512) return s;
  }
  s.n = 0;
  return s;
}

}  // namespace stk

using namespace stk;

// Whether the kernel covers a layer.
STK_API int stk_talking_tokens_ok(int heads, int kv_heads, int kp, int vp, int max_span) {
  if (heads < 1 || kv_heads < 1 || kp % 8 || vp % 8) return 0;
  return tt_shape(heads, kv_heads, kp, vp, max_span).n > 0 ? 1 : 0;
}

// Splits of the key range for T tokens that see at most `keys` keys, and whether every key/value head is a group of its own, which reads
// the keys once per group and of the values only its own: the smallest number of block steps.  splits + 256 * that; 0: not covered.
STK_API int stk_talking_tokens_plan(int T, int heads, int kv_heads, int kp, int vp, int max_span, int keys, int sm_count) {
  int best = 0;
  double cost = 1e30;
  for (int own = 0; own < (max_span < 2 && kv_heads > 1 ? 2 : 1); ++own) {
    const TtShape s = tt_shape(heads, kv_heads, kp, vp, max_span, own ? heads / kv_heads : 0);
    if (s.n == 0 || (own && best == 0)) continue;
    const int groups = (heads + s.hs - 1) / s.hs, tq = max_span < 2 ? 1 : s.n / s.hs;
    const int tiles = ((T + tq - 1) / tq) * groups, blocks = (keys + kTtBlock - 2) / kTtBlock + 1;
    const int held = (s.hs + heads / kv_heads - 1) / (heads / kv_heads);                // key/value heads whose values a group reads
    const double step = static_cast<double>(kv_heads * kp + held * vp) / (kv_heads * (kp + vp));
    for (int n = 1; n <= kTtMaxSplits && n <= blocks; ++n) {
      const int waves = (tiles * n + sm_count - 1) / sm_count;
      const double c = static_cast<double>(waves) * ((blocks + n - 1) / n * step + 1.5) + 0.03 * n;
      if (c < cost - 1e-9) { cost = c; best = n + 256 * own; }
    }
  }
  return best;
}

// Spans of at most max_span tokens.  plan: of stk_talking_tokens_plan.  part: [splits][T][heads][vdim + 2] fp32.
STK_API int stk_talking_tokens(const void* q, const float* gate, const float* sink, const int64_t* positions, const int* tok_req,
                               const int* table, int bt_stride, const void* cache, int row, int k_col, int kp, int vp, int heads, int kv_heads,
                               int vdim, int chunk, float scale, void* out, long long ldo, int out_cols, const int* query_start,
                               const int* req_rows, const int* start_pos, int n_req, const int* first_pos, const int* last_pos, int max_span,
                               long long num_pages, int plan, float* part, int T, int* status, void* stream) {
  if (T <= 0) return 0;
  const int splits = plan & 255;
  TtArgs x;
  x.a = {q, T, gate, sink, positions, tok_req, table, bt_stride, cache, row, k_col, kp, vp, heads, kv_heads, vdim, chunk, scale, out, ldo,
         out_cols};
  const TtShape s = tt_shape(heads, kv_heads, kp, vp, max_span, plan >= 256 ? heads / kv_heads : 0);
  if (!talk_ok(x.a) || s.n == 0 || splits < 1 || splits > kTtMaxSplits || n_req < 1 || num_pages < 1 || row % 8 || kp % 8 || vp % 8 ||
      heads > 65535 || row != k_col + kv_heads * kp || num_pages * kTkPage >= (1ll << 31) ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15))
    return -1;
  const int groups = (heads + s.hs - 1) / s.hs;
  x.hs = s.hs;
  x.tq = max_span < 2 ? 1 : s.n / s.hs;
  x.query_start = query_start; x.req_rows = req_rows; x.start_pos = start_pos; x.n_req = n_req; x.max_span = max_span;
  x.k_pairs = s.k_pairs; x.slots = s.slots;
  x.part = part; x.T = T; x.status = status;
  static_assert(sizeof(TtBars) <= 256, "barrier block");
  CUtensorMap tm;
  if (make_tmap_2d(&tm, cache, 2, num_pages * kTkPage, row, row, kTkPage) != 0) return -3;
  int smem = s.slots * 2 * kTtPanel + tt_fixed(s);
  if (smem < 118 * 1024) smem = 118 * 1024;                          // one CTA per SM: it owns all of tensor memory
  const int tiles = max_span < 2 ? min(T, n_req) : T / x.tq + n_req;
  if (tiles > 65535) return -2;
  const dim3 grid(splits, tiles, groups);
  cudaStream_t st = (cudaStream_t)stream;
  if (s.n == 16) {
    if (cudaFuncSetAttribute(talking_tokens_tc_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -3;
    launch_pdl(talking_tokens_tc_kernel<16>, grid, dim3(kTtThreads), smem, st, tm, x);
  } else {
    if (cudaFuncSetAttribute(talking_tokens_tc_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -3;
    launch_pdl(talking_tokens_tc_kernel<32>, grid, dim3(kTtThreads), smem, st, tm, x);
  }
  launch_pdl(talking_merge_kernel, dim3(T, heads), dim3(128), 0, st, x.a, (const float*)part, splits, first_pos, last_pos, max_span, T);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
