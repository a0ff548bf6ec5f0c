// Latent attention of decode rows and short spans on the 5th-generation tensor cores (bf16): queries in latent space against the
// cached rows, which are key and value for all heads at once.
//
// One CTA per (split of the key range, tile of tokens, group of heads).  The tile's (token, head) pairs are N = 16 or 32 columns:
//
//   loader warp      blocks of 128 rows (two pages) by TMA as panels of 64 columns, in pairs of panels through a ring; an odd last
//                    panel (the rotated part) has two buffers of its own
//   MMA warp         S^T[key, column] = rows . Q^T as the panels arrive; O^T[dim, column] += rows^T . P with the same panels as
//                    MN-major operand, 128 dims at a time, giving each pair of panels back as soon as its dims are done
//   softmax warps    eight, one key and half of the columns per thread: column maxima over the lanes, probabilities to shared memory as bf16 pairs (high parts
//                    and remainders are 2N columns of one product), O rescaled only when a column's maximum grew by more than 2^8
//
// Each CTA writes an unnormalised partial result; latent_merge joins the splits and applies the output gate.  Rows behind the last
// visible key are zeroed in shared memory, so what an earlier owner left in a page cannot reach a sum.  Every mbarrier wait is
// bounded.
#define STK_PDL_CLASS 128
#include "latent_attention.cuh"
#include "warp_reduce.cuh"

namespace stk {

int make_tmap_2d(CUtensorMap* tm, const void* base, int elem_bytes, long long rows, long long cols, long long ld, int box_rows);

constexpr int kLtBlock = 128, kLtPanel = kLtBlock * 128, kLtThreads = 320, kLtMaxPairs = 6;
constexpr float kLtLog2e = 1.4426950408889634f;

struct LtArgs {
  LatArgs l;
  const int* query_start; const int* req_rows; const int* start_pos;
  int n_req, max_span;
  int tq, hs;                            // tokens per tile, heads per group (tq * hs <= N)
  int pairs, tail, slots, v_tiles;       // panel pairs of a row, whether an odd panel follows, ring size, 128-dim tiles
  float* part;                           // [splits][T][H][C + 2]
  int T;
  int* status;
};

struct alignas(8) LtBars {
  uint64_t full[kLtMaxPairs], empty[kLtMaxPairs], tail_full[2], tail_empty[2];
  uint64_t s_full[2], p_full, pv_done, clean;
  uint32_t tmem_base;
  int find[2];
};

__device__ __forceinline__ float lt_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Barrier of the softmax warps that also tells whether every one of them is fine: they leave their loop together.
__device__ __forceinline__ bool lt_bar_all(bool ok) {
  int r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.s32 p, %1, 0;\n\t"
      "barrier.cta.red.and.pred q, 1, 256, p;\n\t"
      "selp.s32 %0, 1, 0, q;\n\t}"
      : "=r"(r) : "r"(ok ? 1 : 0) : "memory");
  return r != 0;
}
__device__ __forceinline__ void lt_bar_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
__device__ __forceinline__ void lt_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
      "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
// 8 or 16 columns of the warp's 32 lanes
template <int C>
__device__ __forceinline__ void lt_ld(uint32_t taddr, uint32_t (&r)[C]) {
  if constexpr (C == 16) {
    tmem_ld_32x16(taddr, r);
  } else {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                 : "r"(taddr));
  }
}
__device__ __forceinline__ void lt_cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

template <int N>
__global__ void __launch_bounds__(kLtThreads, 1)
latent_tokens_tc_kernel(const __grid_constant__ CUtensorMap tm_rows, const LtArgs x) {
  constexpr int kTmemCols = 512;
  extern __shared__ uint8_t smem_raw[];
  const LatArgs& a = x.l;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int q_panels = 2 * x.pairs + x.tail;
  uint8_t* ring = smem;                                             // [slots][2 panels][128 rows x 128 B]
  uint8_t* tails = ring + x.slots * 2 * kLtPanel;                   // [2][128 rows x 128 B] when there is an odd panel
  uint8_t* q_s = tails + (x.tail ? 2 * kLtPanel : 0);               // [q_panels][N x 128 B]
  uint8_t* p_s = q_s + q_panels * N * 128;                          // [2 key panels][2N x 128 B]: high parts, remainders
  LtBars* bars = reinterpret_cast<LtBars*>(p_s + 2 * 2 * N * 128);
  float* smax = reinterpret_cast<float*>(reinterpret_cast<uint8_t*>(bars) + 256);   // [4][N]
  float* m_ref = smax + 4 * N;                                      // [N]
  float* alpha = m_ref + N;                                         // [N]
  int* col_pos = reinterpret_cast<int*>(alpha + N);                 // [N] last key a column sees (-1: padding)
  int* col_row = col_pos + N;                                       // [N] token * heads + head of a column
  int* flags = col_row + N;
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
    for (int s = 0; s < kLtMaxPairs; ++s) {
      mbar_init(&bars->full[s], 1);
      mbar_init(&bars->empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->tail_full[i], 1);
      mbar_init(&bars->tail_empty[i], 1);
      mbar_init(&bars->s_full[i], 1);
    }
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
  const int tok0 = x.query_start[ri] + off, ntok = min(x.tq, x.query_start[ri + 1] - tok0);
  const int p0 = x.start_pos[ri] + off, p_last = p0 + ntok - 1;
  const int blocks = p_last / kLtBlock + 1;
  const int per = (blocks + gridDim.x - 1) / gridDim.x;
  const int b0 = min(blocks, static_cast<int>(blockIdx.x) * per), b1 = min(blocks, b0 + per);
  float* part = x.part + static_cast<long long>(blockIdx.x) * x.T * a.H * (a.C + 2);
  if (b0 >= b1) {
    for (int e = threadIdx.x; e < ntok * nh; e += kLtThreads) {
      float* o = part + (static_cast<long long>(tok0 + e / nh) * a.H + h0 + e % nh) * (a.C + 2);
      o[a.C] = -INFINITY;
      o[a.C + 1] = 0.f;
    }
    return;
  }
  const int* bt = a.table + static_cast<long long>(x.req_rows[ri]) * a.bt_stride;
  auto load_pair = [&](int st, int d, int pg0, int pg1) {
    mbar_expect_tx(&bars->full[st], 2 * kLtPanel);
    uint8_t* dst = ring + st * 2 * kLtPanel;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      tma_load_2d(dst + j * kLtPanel, &tm_rows, &bars->full[st], (2 * d + j) * 64, pg0 * kLatPage);
      tma_load_2d(dst + j * kLtPanel + kLtPanel / 2, &tm_rows, &bars->full[st], (2 * d + j) * 64, pg1 * kLatPage);
    }
  };
  auto load_tail = [&](int st, int pg0, int pg1) {
    mbar_expect_tx(&bars->tail_full[st], kLtPanel);
    tma_load_2d(tails + st * kLtPanel, &tm_rows, &bars->tail_full[st], 2 * x.pairs * 64, pg0 * kLatPage);
    tma_load_2d(tails + st * kLtPanel + kLtPanel / 2, &tm_rows, &bars->tail_full[st], 2 * x.pairs * 64, pg1 * kLatPage);
  };
  auto page_of = [&](int lp) { return lp <= p_last / kLatPage ? max(bt[lp], 0) : 0; };
  if (warp == 8 && lane == 0) {
    // the first block is on its way while the queries are laid out
    const int pg0 = page_of(2 * b0), pg1 = page_of(2 * b0 + 1);
    for (int d = 0; d < x.pairs; ++d) load_pair(d, d, pg0, pg1);
    if (x.tail) load_tail(0, pg0, pg1);
  }
  if (warp == 9) {
    tmem_alloc(&bars->tmem_base, kTmemCols);
    tmem_relinquish();
  }
  __syncwarp();
  // latent parts of the queries, straight to their places
  for (int n = warp; n < N; n += kLtThreads / 32) {
    const int q = n / x.hs, hh = n - q * x.hs;
    const bool valid = q < ntok && hh < nh;
    const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(a.qa) + (valid ? (tok0 + q) * a.ldqa + (h0 + hh) * a.cp : 0);
    for (int cc = lane; cc < q_panels * 8; cc += 32) {
      uint8_t* dst = q_s + (cc >> 3) * (N * 128) + n * 128 + (((cc & 7) ^ (n & 7)) << 4);
      if (valid && cc * 8 < a.rot_off) lt_cp16(dst, src + cc * 8);
      else if (!valid || cc * 8 >= a.rot_off + a.R) *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
    }
    if (lane == 0) {
      col_pos[n] = valid ? p0 + q : -1;
      col_row[n] = (tok0 + q) * a.H + h0 + hh;
      m_ref[n] = -INFINITY;
    }
  }
  // cos and sin of the tile's positions (in the probabilities' memory, which comes later)
  const int half = a.R >> 1;
  float2* cs = reinterpret_cast<float2*>(p_s);
  const bool table_fits = ntok * half * 8 <= 2 * 2 * N * 128;
  if (table_fits)
    for (int e = threadIdx.x; e < ntok * half; e += kLtThreads) cs[e] = cos_sin_split(p0 + e / half, a.freq[e % half], a.freq[half + e % half]);
  if (threadIdx.x < 2) flags[threadIdx.x] = 0;
  __syncthreads();
  {
    const int chunks = (a.R + 7) / 8;
    for (int e = threadIdx.x; e < N * chunks; e += kLtThreads) {
      const int n = e / chunks, rc = e - n * chunks, cc = (a.rot_off >> 3) + rc;
      if (col_pos[n] < 0) continue;
      const int q = n / x.hs;
      const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(a.qr) + (tok0 + q) * a.ldqr + (h0 + n - q * x.hs) * a.R + rc * 8;
      uint4 v = make_uint4(0, 0, 0, 0);
      __nv_bfloat162* o = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int k = rc * 4 + j;
        if (k < half) {
          const float2 w = table_fits ? cs[q * half + k] : cos_sin_split(p0 + q, a.freq[k], a.freq[half + k]);
          const float u = bf16_to_f(src[2 * j]), y = bf16_to_f(src[2 * j + 1]);
          o[j] = __floats2bfloat162_rn(u * w.x - y * w.y, y * w.x + u * w.y);
        }
      }
      *reinterpret_cast<uint4*>(q_s + (cc >> 3) * (N * 128) + n * 128 + (((cc & 7) ^ (n & 7)) << 4)) = v;
    }
  }
  asm volatile("cp.async.commit_group;\n\tcp.async.wait_group 0;" ::: "memory");
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_base;                            // scores: two buffers of N columns; outputs from column 2N on
  const uint32_t tmem_o = tmem + 2 * N;
  const bool ragged = b1 == blocks && (p_last + 1) % kLtBlock != 0;
  // scores of the next block may be formed before this block's output when the ring holds two blocks
  const bool ahead = x.slots >= 2 * x.pairs;

  if (warp == 8) {
    // ------------------------------- loader -------------------------------
    bool ok = true;
    int seq = x.pairs, done_b = b0 + 1;
    if (lane == 0) {
      for (int b = b0 + 1; b < b1 && ok; ++b) {
        const int pg0 = page_of(2 * b), pg1 = page_of(2 * b + 1);
        for (int d = 0; d < x.pairs; ++d, ++seq) {
          const int st = seq % x.slots;
          if (seq >= x.slots) ok = mbar_wait(&bars->empty[st], ((seq / x.slots) - 1) & 1, x.status, 900);
          if (!ok) break;
          load_pair(st, d, pg0, pg1);
        }
        if (ok && x.tail) {
          const int i = b - b0, st = i & 1;
          if (i >= 2) ok = mbar_wait(&bars->tail_empty[st], ((i >> 1) - 1) & 1, x.status, 901);
          if (!ok) break;
          load_tail(st, pg0, pg1);
          done_b = b + 1;
        }
      }
    }
    ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
    if (ok && ragged) {
      // the last block's rows behind the last key
      const int i = b1 - 1 - b0, row0 = (p_last + 1) % kLtBlock;
      for (int d = 0; d < x.pairs && ok; ++d) {
        const int s = i * x.pairs + d, st = s % x.slots;
        ok = mbar_wait(&bars->full[st], (s / x.slots) & 1, x.status, 902);
        for (int e = row0 * 8 + lane; e < kLtBlock * 8; e += 32) {
          *reinterpret_cast<uint4*>(ring + st * 2 * kLtPanel + e * 16) = make_uint4(0, 0, 0, 0);
          *reinterpret_cast<uint4*>(ring + (st * 2 + 1) * kLtPanel + e * 16) = make_uint4(0, 0, 0, 0);
        }
      }
      if (ok && x.tail) {
        ok = mbar_wait(&bars->tail_full[i & 1], (i >> 1) & 1, x.status, 903);
        for (int e = row0 * 8 + lane; e < kLtBlock * 8; e += 32)
          *reinterpret_cast<uint4*>(tails + (i & 1) * kLtPanel + e * 16) = make_uint4(0, 0, 0, 0);
      }
      fence_proxy_async();
      __syncwarp();
      if (ok && lane == 0) mbar_arrive(&bars->clean);
    }
    if (!ok && lane == 0) {
      // leave no copy in flight: what was asked for lands before the CTA's shared memory goes away
      for (int s = max(0, seq - x.slots); s < seq; ++s) mbar_wait(&bars->full[s % x.slots], (s / x.slots) & 1, nullptr, 0);
      for (int i = max(0, done_b - b0 - 2); x.tail && i < done_b - b0; ++i) mbar_wait(&bars->tail_full[i & 1], (i >> 1) & 1, nullptr, 0);
    }
    __syncwarp();
  } else if (warp == 9) {
    // ------------------------------- MMA issuer -------------------------------
    constexpr uint32_t kIdescS = umma_idesc(1u, 1u, 128, N);
    constexpr uint32_t kIdescO = umma_idesc(1u, 1u, 128, 2 * N) | (1u << 15);             // A is MN-major
    constexpr uint32_t kStep = kLtPanel >> 4, kQStep = (N * 128) >> 4;                    // panels in descriptor units
    const uint32_t lead = elect_one() ? 1u : 0u, tm = __shfl_sync(0xffffffffu, tmem, 0);
    const uint32_t k_lo = desc_lo(smem_u32(ring)), v_lo = desc_lo(smem_u32(ring), kLtPanel), t_lo = desc_lo(smem_u32(tails));
    const uint32_t q_lo = desc_lo(smem_u32(q_s)), p_lo = desc_lo(smem_u32(p_s));
    struct At { int slot; uint32_t par; };
    auto ahead_of = [&](At c, int n) {
      c.slot += n;
      if (c.slot >= x.slots) { c.slot -= x.slots; c.par ^= 1u; }
      return c;
    };
    auto scores = [&](int b, At c) {
      const int i = b - b0;
      if (ragged && b == b1 - 1) {
        if (!mbar_wait(&bars->clean, 0, x.status, 910)) return false;
      }
      const uint32_t d0 = tm + (i & 1) * N;
      for (int d = 0; d < x.pairs; ++d) {
        const At p = ahead_of(c, d);
        if (!mbar_wait(&bars->full[p.slot], p.par, x.status, 911)) return false;
        tc_fence_after();
        const uint32_t al = k_lo + p.slot * 2 * kStep, bl = q_lo + d * 2 * kQStep;
#pragma unroll
        for (int ks = 0; ks < 8; ++ks)
          mma_ss(d0, al + (ks >> 2) * kStep + 2 * (ks & 3), bl + (ks >> 2) * kQStep + 2 * (ks & 3), kIdescS,
                 ks > 0 ? 1u : (d > 0 ? 1u : 0u), lead);
        if (d >= x.v_tiles) mma_commit(&bars->empty[p.slot], lead);
      }
      if (x.tail) {
        if (!mbar_wait(&bars->tail_full[i & 1], (i >> 1) & 1, x.status, 912)) return false;
        tc_fence_after();
        const uint32_t al = t_lo + (i & 1) * kStep, bl = q_lo + 2 * x.pairs * kQStep;
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) mma_ss(d0, al + 2 * ks, bl + 2 * ks, kIdescS, ks > 0 ? 1u : (x.pairs > 0 ? 1u : 0u), lead);
        mma_commit(&bars->tail_empty[i & 1], lead);
      }
      mma_commit(&bars->s_full[i & 1], lead);
      return true;
    };
    At cur{0, 0u};                                                  // first pair of block b
    bool ok = scores(b0, cur);
    for (int b = b0; b < b1 && ok; ++b) {
      const int i = b - b0;
      const At next = ahead_of(cur, x.pairs);
      if (ahead && b + 1 < b1) ok = scores(b + 1, next);
      if (ok) ok = mbar_wait(&bars->p_full, i & 1, x.status, 913);
      if (!ok) break;
      tc_fence_after();
      for (int j = 0; j < x.v_tiles; ++j) {
        const int st = ahead_of(cur, j).slot;
        const uint32_t al = v_lo + st * 2 * kStep, dj = tm + 2 * N + j * 2 * N;
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          mma_ss(dj, al + kk * 128, p_lo + (kk >> 2) * 2 * kQStep + 2 * (kk & 3), kIdescO, kk > 0 ? 1u : (i > 0 ? 1u : 0u), lead);
        mma_commit(&bars->empty[st], lead);
      }
      mma_commit(&bars->pv_done, lead);
      if (!ahead && b + 1 < b1) ok = scores(b + 1, next);
      cur = next;
    }
    __syncwarp();
  } else {
    // ------------------------------- softmax -------------------------------
    constexpr int NH = N / 2;                                       // columns of this thread
    const int row = (warp & 3) * 32 + lane, c0 = (warp >> 2) * NH;
    const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const float c_in = a.scale * kLtLog2e;
    float l[NH];
#pragma unroll
    for (int n = 0; n < NH; ++n) l[n] = 0.f;
    bool ok = true;
    for (int b = b0; b < b1; ++b) {
      const int i = b - b0, key = b * kLtBlock + row;
      ok = ok && mbar_wait(&bars->s_full[i & 1], (i >> 1) & 1, x.status, 920);
      tc_fence_after();
      float v[NH], keep[NH];
      {
        uint32_t r[NH];
        lt_ld<NH>(tmem + (i & 1) * N + c0 + lanes, r);
        tmem_ld_wait();
#pragma unroll
        for (int n = 0; n < NH; ++n) v[n] = __uint_as_float(r[n]) * c_in;
        if (b * kLtBlock + kLtBlock - 1 > p0) {
#pragma unroll
          for (int n = 0; n < NH; ++n)
            if (key > col_pos[c0 + n]) v[n] = -INFINITY;
        }
      }
#pragma unroll
      for (int n = 0; n < NH; ++n) keep[n] = v[n];
      bfly_reduce_store<NH, true>(v, smax + (warp & 3) * N + c0, lane);
      ok = lt_bar_all(ok);
      if (!ok) break;
      if (threadIdx.x == 0) flags[(i + 1) & 1] = 0;
      if (threadIdx.x < N) {
        const int n = threadIdx.x;
        const float bm = fmaxf(fmaxf(smax[n], smax[N + n]), fmaxf(smax[2 * N + n], smax[3 * N + n]));
        const float mo = m_ref[n];
        float f = 1.f;
        if (bm > mo + 8.f || (mo == -INFINITY && bm > -INFINITY)) {
          f = mo == -INFINITY ? 0.f : lt_ex2(mo - bm);
          m_ref[n] = bm;
          flags[i & 1] = 1;
        }
        alpha[n] = f;
      }
      lt_bar_sync();
      if (i > 0) {
        // the previous product has read the probabilities and finished its output
        ok = mbar_wait(&bars->pv_done, (i - 1) & 1, x.status, 921);
        if (!ok) continue;
        tc_fence_after();
      }
      if (flags[i & 1]) {
#pragma unroll
        for (int n = 0; n < NH; ++n) l[n] *= alpha[c0 + n];
        if (i > 0) {
          // high parts for the first four warps, remainders for the others
          const uint32_t to = tmem_o + (warp >> 2) * N + lanes;
          for (int j = 0; j < x.v_tiles; ++j)
#pragma unroll
            for (int c = 0; c < N; c += 16) {
              uint32_t o[16];
              tmem_ld_32x16(to + j * 2 * N + c, o);
              tmem_ld_wait();
#pragma unroll
              for (int k = 0; k < 16; ++k) o[k] = __float_as_uint(__uint_as_float(o[k]) * alpha[c + k]);
              lt_st16(to + j * 2 * N + c, o);
            }
          asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        }
      }
      uint8_t* dst = p_s + (row >> 6) * (2 * N * 128) + c0 * 128 + (row & 7) * 2;
      const int chunk = (row & 63) >> 3;
#pragma unroll
      for (int n = 0; n < NH; ++n) {
        const float mr = m_ref[c0 + n];
        const float p = mr == -INFINITY ? 0.f : lt_ex2(keep[n] - mr);
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
    if (ok) ok = mbar_wait(&bars->pv_done, (b1 - 1 - b0) & 1, x.status, 922);
    tc_fence_after();
    bfly_reduce_store<NH, false>(l, smax + (warp & 3) * N + c0, lane);
    lt_bar_sync();
    if (ok) {
      // the two halves of the warps take every other 128 dims
      for (int j = warp >> 2; j < x.v_tiles; j += 2) {
        const int d = j * 128 + row;
#pragma unroll
        for (int c = 0; c < N; c += 16) {
          uint32_t u[16], w[16];
          tmem_ld_32x16(tmem_o + j * 2 * N + c + lanes, u);
          tmem_ld_32x16(tmem_o + j * 2 * N + N + c + lanes, w);
          tmem_ld_wait();
          if (d < a.C) {
#pragma unroll
            for (int k = 0; k < 16; ++k)
              if (col_pos[c + k] >= 0)
                part[static_cast<long long>(col_row[c + k]) * (a.C + 2) + d] = __uint_as_float(u[k]) + __uint_as_float(w[k]);
          }
        }
      }
      if (threadIdx.x < N && col_pos[threadIdx.x] >= 0) {
        const int n = threadIdx.x;
        float* o = part + static_cast<long long>(col_row[n]) * (a.C + 2);
        o[a.C] = m_ref[n];
        o[a.C + 1] = (smax[n] + smax[N + n]) + (smax[2 * N + n] + smax[3 * N + n]);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    tmem_dealloc(tmem, kTmemCols);
  }
}

// One CTA per (token, head, part of the dims): joins the splits, normalises, gates; zeros behind the latent's dimensions and for padding tokens.
constexpr int kLtMaxSplits = 64;

__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part, int splits, const float* __restrict__ gate, long long ldg,
                    const int64_t* __restrict__ positions, const int* __restrict__ tok_req, const int* __restrict__ first_pos,
                    const int* __restrict__ last_pos, int max_span, int T, int H, int C, int cp, __nv_bfloat16* __restrict__ out,
                    long long ldo) {
  __shared__ float wt[kLtMaxSplits];
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const int h = blockIdx.y;
  __nv_bfloat16* o = out + t * ldo + h * cp;
  const int d0 = blockIdx.z * blockDim.x + threadIdx.x, dstep = gridDim.z * blockDim.x;
  if (tok_req[t] < 0 || positions[t] < 0) {
    for (int d = d0; d < cp; d += dstep) o[d] = __float2bfloat16(0.f);
    return;
  }
  if (last_pos[t] - first_pos[t] + 1 > max_span) return;
  const long long step = static_cast<long long>(T) * H * (C + 2);
  const float* p = part + (t * H + h) * (C + 2);
  if (threadIdx.x < 32) {
    // the splits' weights: two per lane
    float m[2], l[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int s = threadIdx.x + i * 32;
      m[i] = s < splits ? p[s * step + C] : -INFINITY;
      l[i] = s < splits ? p[s * step + C + 1] : 0.f;
    }
    const float mx = warp_max(fmaxf(m[0], m[1]));
    float sum = 0.f, f[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      f[i] = m[i] == -INFINITY ? 0.f : lt_ex2(m[i] - mx);
      sum = fmaf(f[i], l[i], sum);
    }
    const float g = (gate != nullptr ? lat_sigmoid(gate[t * ldg + h]) : 1.f) / warp_sum(sum);
    wt[threadIdx.x] = f[0] * g;
    wt[threadIdx.x + 32] = f[1] * g;
  }
  __syncthreads();
  for (int d = d0; d < cp; d += dstep) {
    float v = 0.f;
    if (d < C) {
      // a split without keys left its columns unwritten
#pragma unroll 16
      for (int s = 0; s < splits; ++s) {
        const float w = wt[s];
        v = fmaf(w, w != 0.f ? p[s * step + d] : 0.f, v);
      }
    }
    o[d] = __float2bfloat16(v);
  }
}

struct LtShape {
  int pairs, tail, v_tiles, slots;
};
static LtShape lt_shape(int C, int row, int n) {
  LtShape s;
  const int panels = (row + 63) / 64;
  s.v_tiles = (C + 127) / 128;
  s.pairs = panels / 2;
  s.tail = panels & 1;
  if (s.pairs < s.v_tiles) { s.pairs = s.v_tiles; s.tail = 0; }        // the values reach into the odd panel
  const int fixed = (2 * s.pairs + s.tail) * n * 128 + 4 * n * 128 + (s.tail ? 2 * kLtPanel : 0) + 256 + 8 * n * 4 + 64 + 1024;
  s.slots = (227 * 1024 - fixed) / (2 * kLtPanel);
  if (s.slots > kLtMaxPairs) s.slots = kLtMaxPairs;
  return s;
}

}  // namespace stk

using namespace stk;

// Columns (16 or 32) the kernel would use for a layer and span length, 0 when it does not cover the layer.
STK_API int stk_latent_tokens_columns(int heads, int kv_rank, int row, int max_span) {
  if (heads < 1 || kv_rank < 1 || row % 8 || kv_rank > 512) return 0;
  const int groups = (heads + 31) / 32, hs = (heads + groups - 1) / groups;
  const int n = hs <= 16 && (max_span < 2 || 2 * hs > 16) ? 16 : 32;
  const LtShape s = lt_shape(kv_rank, row, n);
  return s.slots >= s.pairs ? n : 0;
}

// Splits of the key range for T tokens with contexts of at most `context` tokens: the smallest number of block steps.
STK_API int stk_latent_tokens_splits(int T, int heads, int max_span, int context, int sm_count) {
  const int groups = (heads + 31) / 32, hs = (heads + groups - 1) / groups;
  const int tq = max_span < 2 ? 1 : (hs <= 32 ? 32 / hs : 1);
  const int tiles = ((T + tq - 1) / tq) * groups;
  const int blocks = context / kLtBlock + 1;
  int best = 1;
  double cost = 1e30;
  for (int s = 1; s <= kLtMaxSplits && s <= blocks; ++s) {
    const int waves = (tiles * s + sm_count - 1) / sm_count;
    const double c = static_cast<double>(waves) * ((blocks + s - 1) / s + 1.5) + 0.03 * s;
    if (c < cost - 1e-9) { cost = c; best = s; }
  }
  return best;
}

// Spans of at most max_span tokens.  part: [splits][T][heads][kv_rank + 2] fp32.
STK_API int stk_latent_tokens(const void* qa, long long ldqa, int cp, const void* qr, long long ldqr, const float* gate, long long ldg,
                              const int64_t* positions, const int* tok_req, const int* table, int bt_stride, const void* cache,
                              int row, int rot_off, const float* freq, int heads, int kv_rank, int rot, float scale, void* out,
                              long long ldo, const int* query_start, const int* req_rows, const int* start_pos, int n_req,
                              const int* first_pos, const int* last_pos, int max_span, long long num_pages, int splits, float* part,
                              int T, int* status, void* stream) {
  if (T <= 0) return 0;
  LtArgs x;
  x.l = lat_args(qa, ldqa, cp, qr, ldqr, gate, ldg, positions, tok_req, table, bt_stride, cache, row, rot_off, freq, heads, kv_rank,
                 rot, scale, out, ldo);
  const int n = stk_latent_tokens_columns(heads, kv_rank, row, max_span);
  if (!lat_ok(x.l) || n == 0 || splits < 1 || splits > kLtMaxSplits || n_req < 1 || num_pages < 1 || ldqa % 8 || cp % 8 || rot_off % 8 || heads > 65535 ||
      ((reinterpret_cast<uintptr_t>(qa) | reinterpret_cast<uintptr_t>(cache)) & 15))
    return -1;
  const LtShape s = lt_shape(kv_rank, row, n);
  const int groups = (heads + 31) / 32;
  x.hs = (heads + groups - 1) / groups;
  x.tq = max_span < 2 ? 1 : n / x.hs;
  x.query_start = query_start; x.req_rows = req_rows; x.start_pos = start_pos; x.n_req = n_req; x.max_span = max_span;
  x.pairs = s.pairs; x.tail = s.tail; x.slots = s.slots; x.v_tiles = s.v_tiles;
  x.part = part; x.T = T; x.status = status;
  static_assert(sizeof(LtBars) <= 256, "barrier block");
  CUtensorMap tm;
  if (make_tmap_2d(&tm, cache, 2, num_pages * kLatPage, row, row, kLatPage) != 0) return -3;
  int smem = s.slots * 2 * kLtPanel + (s.tail ? 2 * kLtPanel : 0) + (2 * s.pairs + s.tail) * n * 128 + 4 * n * 128 + 256 + 8 * n * 4 +
             64 + 1024;
  if (smem < 118 * 1024) smem = 118 * 1024;                          // one CTA per SM: it owns all of tensor memory
  const int tiles = max_span < 2 ? min(T, n_req) : T / x.tq + n_req;
  if (tiles > 65535) return -2;
  const dim3 grid(splits, tiles, groups);
  cudaStream_t st = (cudaStream_t)stream;
  if (n == 16) {
    if (cudaFuncSetAttribute(latent_tokens_tc_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -3;
    launch_pdl(latent_tokens_tc_kernel<16>, grid, dim3(kLtThreads), smem, st, tm, x);
  } else {
    if (cudaFuncSetAttribute(latent_tokens_tc_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -3;
    launch_pdl(latent_tokens_tc_kernel<32>, grid, dim3(kLtThreads), smem, st, tm, x);
  }
  // few rows: every 128 dims get a CTA of their own (each waits for as many loads as there are splits)
  const int z = static_cast<long long>(T) * heads < 1024 ? (cp + 127) / 128 : 1;
  launch_pdl(latent_merge_kernel, dim3(T, heads, z), dim3(128), 0, st, (const float*)part, splits, gate, ldg, positions, tok_req, first_pos,
             last_pos, max_span, T, heads, kv_rank, cp, (__nv_bfloat16*)out, ldo);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
