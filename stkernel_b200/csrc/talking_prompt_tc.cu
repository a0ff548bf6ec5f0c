// Talking-heads attention of prompt portions on the 5th-generation tensor cores (bf16).  Mixed queries meet the keys of all key/value heads
// side by side, so a head's scores contract kv_heads * kp columns; its values are those of its own key/value head.
//
//   talking_rows         the cached rows that a request's long span can see, copied out of their pages into one matrix; each request
//                        starts on a 128-row border and is padded with zero rows to the next one
//   talking_prompt_tc    one CTA per SM takes (tile of 128 query tokens, head) after (tile, head), the longest first, over blocks of 128 keys
//
//     loader warp      the tile's queries (kept in shared memory; where they are too wide, a panel at a time with the keys) and, through a
//                      ring of 16 KB panels [128 rows x 64 columns], keys and values in the order in which they are used; the next tile's
//                      operands arrive while the last blocks of this one are weighted and written
//     MMA warp         S[query, key] = Q . K^T, then O[query, v] += P . V with P read from tensor memory.  Blocks take turns between two
//                      sets of accumulators, so one block's softmax runs under the products of the next
//     softmax warps    eight per set, half of a row's scores per thread: running maximum (O rescaled only when a row's maximum grew by more than 2^8),
//                      probabilities written over the scores as bf16 pairs (high part and remainder, two products)
//
// The two sets hold partial results of the same rows with maxima and denominators of their own; they are joined at the end.
// TMEM: per set 128 columns of scores / probabilities and up to 128 of O.  Every mbarrier wait is bounded.
#define STK_PDL_CLASS 8
#include "latent_attention.cuh"
#include "talking_attention.cuh"

namespace stk {

int make_tmap_2d(CUtensorMap* tm, const void* base, int elem_bytes, long long rows, long long cols, long long ld, int box_rows);

constexpr int kTpTile = 128, kTpPanel = kTpTile * 128, kTpThreads = 608, kTpMaxSlots = 12, kTpMaxQ = 10;
constexpr float kTpLog2e = 1.4426950408889634f;

struct alignas(8) TpBars {
  uint64_t q_full, q_empty, full[kTpMaxSlots], empty[kTpMaxSlots];
  uint64_t s_full[2], p_full[2], o_full, o_empty;
  uint32_t tmem_base;
  float row_max[4 * 128];                                          // [set][half][row]
};
constexpr int kTpBarBytes = 3072;

struct TpArgs {
  TalkArgs a;
  const int* query_start; const int* start_pos;
  int n_req, min_span;
  int k_panels, v_panels, q_kept;        // panels of 64 columns; whether the queries stay in shared memory
  int slots, T;
  int* status;
};


__device__ __forceinline__ void tp_ld8(uint32_t taddr, uint32_t (&r)[8]) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
               : "r"(taddr));
}
__device__ __forceinline__ void tp_st8(uint32_t taddr, const uint32_t (&r)[8]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};"
               ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7])
               : "memory");
}
__device__ __forceinline__ void tp_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ float tp_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Barrier `id` of `n` threads that also tells whether all of them are fine.
__device__ __forceinline__ bool tp_bar_all(int id, bool ok, int n = 256) {
  int r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.s32 p, %1, 0;\n\t"
      "barrier.cta.red.and.pred q, %2, %3, p;\n\t"
      "selp.s32 %0, 1, 0, q;\n\t}"
      : "=r"(r) : "r"(ok ? 1 : 0), "r"(id), "r"(n) : "memory");
  return r != 0;
}
// First row that a span starting at `start` needs: its chunk's first position, on a 128-row border.
__host__ __device__ inline int tp_base(int chunk, int start) { return chunk > 0 ? start / chunk * chunk / kTpTile * kTpTile : 0; }

// kTpParts CTAs per 128 rows of the gathered matrix.
constexpr int kTpParts = 32;
__global__ void __launch_bounds__(256)
talking_rows_kernel(const int* __restrict__ query_start, const int* __restrict__ req_rows, const int* __restrict__ start_pos, int n_req,
                    int min_span, int chunk, const int* __restrict__ table, int bt_stride, const __nv_bfloat16* __restrict__ cache, int row,
                    __nv_bfloat16* __restrict__ out) {
  __shared__ int found[4];
  pdl_wait();
  pdl_trigger();
  if (threadIdx.x == 0) {
    int left = blockIdx.x, ri = -1, ctx = 0, first = 0;
    for (int i = 0; i < n_req; ++i) {
      const int n = query_start[i + 1] - query_start[i];
      if (n < min_span) continue;
      const int base = tp_base(chunk, start_pos[i]);
      ctx = start_pos[i] + n;
      const int tiles = (ctx - base + kTpTile - 1) / kTpTile;
      first = start_pos[i];
      if (left < tiles) { ri = i; left = base + left * kTpTile; break; }
      left -= tiles;
    }
    found[0] = ri; found[1] = left; found[2] = ctx; found[3] = chunk > 0 ? first / chunk * chunk : 0;
  }
  __syncthreads();
  const int ri = found[0], j0 = found[1], ctx = found[2], lo = found[3];
  const int chunks = row >> 3;
  constexpr int kRows = kTpTile / kTpParts;
  const int part = blockIdx.y * kRows;
  uint4* dst = reinterpret_cast<uint4*>(out + (static_cast<long long>(blockIdx.x) * kTpTile + part) * row);
  const int* bt = ri >= 0 ? table + static_cast<long long>(req_rows[ri]) * bt_stride : nullptr;
  for (int e = threadIdx.x; e < kRows * chunks; e += blockDim.x) {
    const int r = e / chunks, c = e - r * chunks, j = j0 + part + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (ri >= 0 && j >= lo && j < ctx) {
      const int page = bt[j / kTkPage];
      if (page >= 0) v = *reinterpret_cast<const uint4*>(cache + (static_cast<long long>(page) * kTkPage + j % kTkPage) * row + c * 8);
    }
    dst[e] = v;
  }
}

// The n-th (tile, head) of this CTA; nb 0 when there is none.
struct TpItem { int h, row0, n_tok, first, last, base, seg, b0, nb; };
__device__ __forceinline__ TpItem tp_item(const TpArgs& x, int n) {
  TpItem t = {};
  // every other round in reverse, so that no CTA always has the longer ones
  const long long w = static_cast<long long>(n) * gridDim.x + ((n & 1) ? gridDim.x - 1 - blockIdx.x : blockIdx.x);
  int left = static_cast<int>(w / x.a.H), seg = 0;
  t.h = static_cast<int>(w % x.a.H);
  for (int i = 0; i < x.n_req; ++i) {
    const int q0 = x.query_start[i], span = x.query_start[i + 1] - q0;
    if (span < x.min_span) continue;
    const int tiles = (span + kTpTile - 1) / kTpTile, start = x.start_pos[i], base = tp_base(x.a.chunk, start);
    if (left < tiles) {
      const int off = (tiles - 1 - left) * kTpTile;                // the longest contexts of a request first
      t.row0 = q0 + off;
      t.n_tok = min(kTpTile, span - off);
      t.first = start + off;
      t.last = t.first + t.n_tok - 1;
      t.base = base;
      t.seg = seg;
      t.b0 = (talk_first(x.a, t.first) - base) / kTpTile;
      t.nb = (t.last - base) / kTpTile + 1 - t.b0;                 // blocks of gathered rows
      return t;
    }
    left -= tiles;
    seg += (start + span - base + kTpTile - 1) / kTpTile * kTpTile;
  }
  return t;
}

__global__ void __launch_bounds__(kTpThreads, 1)
talking_prompt_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_r, const TpArgs x) {
  extern __shared__ __align__(1024) uint8_t smem[];
  const TalkArgs& a = x.a;
  if ((smem_u32(smem) & 1023) != 0) {                              // the panels' swizzle needs it; there is no room to round up
    pdl_wait();
    set_status(x.status, kBadIndex, 859);
    return;
  }
  const int kp = x.k_panels;
  uint8_t* q_s = smem;                                             // [kp][128 rows x 128 B] when the queries are kept
  uint8_t* ring = q_s + (x.q_kept ? kp * kTpPanel : 0);            // [slots][128 rows x 128 B]
  TpBars* bars = reinterpret_cast<TpBars*>(ring + x.slots * kTpPanel);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&bars->q_full, 1);
    mbar_init(&bars->q_empty, 1);
    for (int s = 0; s < kTpMaxSlots; ++s) {
      mbar_init(&bars->full[s], 1);
      mbar_init(&bars->empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->s_full[i], 1);
      mbar_init(&bars->p_full[i], 8);
    }
    mbar_init(&bars->o_full, 1);
    mbar_init(&bars->o_empty, 16);
    fence_barrier_init();
  }
  if (warp == 17) {
    tmem_alloc(&bars->tmem_base, 512);
    tmem_relinquish();
  }
  pdl_wait();
  pdl_trigger();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_base;                           // scores of set i: i * 128; outputs: 256 + i * 128

  if (warp == 16 || warp == 18) {
    // ------------------------------- loader -------------------------------
    if (lane == 0) {
      bool ok = true, wrapped = false, turn = warp == 16;          // the two loaders take the panels in turn
      int asked = 0, slot = 0;                                     // tiles whose queries were asked for; the next slot and
      uint32_t par = 1u;                                           // the parity of its release (a fresh barrier passes for 1)
      const int slots = x.slots;
      auto load = [&](const CUtensorMap* tm, int col, int y) {
        if (turn) {
          uint64_t* full = bars->full + slot;
          if (!mbar_wait(bars->empty + slot, par, x.status, 860)) { ok = false; return; }
          mbar_expect_tx(full, kTpPanel);
          tma_load_2d(ring + slot * kTpPanel, tm, full, col, y);
        }
        turn = !turn;
        if (++slot == slots) { slot = 0; par ^= 1u; wrapped = true; }
      };
      for (int items = 0; ok; ++items) {
        const TpItem t = tp_item(x, items);
        if (t.nb == 0) break;
        const int qy = t.h * x.T + t.row0, vc = t.h / (a.H / a.G) * a.vp;
        const int y0 = t.seg + t.b0 * kTpTile;
        auto keys = [&](int b, int j0, int j1) {
          for (int j = j0; j < j1 && ok; ++j) {
            if (!x.q_kept) load(&tm_q, j * 64, qy);
            if (ok) load(&tm_r, a.k_col + j * 64, y0 + b * kTpTile);
          }
        };
        int ahead = 0;
        if (x.q_kept) {
          // as many keys as the ring takes without the products' help, then the queries in place of the previous tile's
          ahead = min(kp, x.slots);
          keys(0, 0, ahead);
          if (ok && items > 0 && warp == 16) ok = mbar_wait(&bars->q_empty, (items - 1) & 1, x.status, 861);
          if (!ok) break;
          if (warp == 16) {
            mbar_expect_tx(&bars->q_full, kp * kTpPanel);
            for (int p = 0; p < kp; ++p) tma_load_2d(q_s + p * kTpPanel, &tm_q, &bars->q_full, p * 64, qy);
            ++asked;
          }
        }
        keys(0, ahead, kp);
        if (t.nb > 1) keys(1, 0, kp);
        for (int b = 0; b < t.nb && ok; ++b) {
          for (int j = 0; j < x.v_panels && ok; ++j) load(&tm_r, vc + j * 64, y0 + b * kTpTile);
          if (b + 2 < t.nb) keys(b + 2, 0, kp);
        }
      }
      if (!ok) {
        // leave no copy in flight: what was asked for lands before the CTA's shared memory goes away
        if (asked > 0) mbar_wait(&bars->q_full, (asked - 1) & 1, nullptr, 0);
        for (int s = 0; s < (wrapped ? slots : slot); ++s) mbar_wait(&bars->full[s], s < slot ? par ^ 1u : par, nullptr, 0);
      }
    }
    __syncwarp();
  } else if (warp == 17) {
    // ------------------------------- MMA issuer -------------------------------
    const uint32_t lead = elect_one() ? 1u : 0u, tm = __shfl_sync(0xffffffffu, tmem, 0);
    constexpr uint32_t kIdescS = umma_idesc(1u, 1u, 128, 128);
    constexpr uint32_t kIdescO1 = umma_idesc(1u, 1u, 128, 64) | (1u << 16), kIdescO2 = umma_idesc(1u, 1u, 128, 128) | (1u << 16);
    constexpr uint32_t kStep = kTpPanel >> 4;                      // a panel in descriptor units
    const uint32_t q_lo = desc_lo(smem_u32(q_s)), k_lo = desc_lo(smem_u32(ring)), v_lo = desc_lo(smem_u32(ring), kTpPanel);
    int slot = 0;
    uint32_t par = 0u, used0 = 0u, used1 = 0u;                     // blocks that went through each set, modulo 2
    bool ok = true;
    auto next = [&]() {
      if (++slot == x.slots) { slot = 0; par ^= 1u; }
    };
    auto scores = [&](int i) {
      for (int j = 0; j < kp; ++j) {
        uint32_t al = q_lo + j * kStep;
        int q_slot = -1;
        if (!x.q_kept) {
          if (!mbar_wait(&bars->full[slot], par, x.status, 862)) return false;
          al = k_lo + slot * kStep;
          q_slot = slot;
          next();
        }
        if (!mbar_wait(&bars->full[slot], par, x.status, 863)) return false;
        tc_fence_after();
        const uint32_t bl = k_lo + slot * kStep;
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) mma_ss(tm + i * 128, al + 2 * ks, bl + 2 * ks, kIdescS, ks > 0 ? 1u : (j > 0 ? 1u : 0u), lead);
        if (q_slot >= 0) mma_commit(&bars->empty[q_slot], lead);
        mma_commit(&bars->empty[slot], lead);
        next();
      }
      mma_commit(&bars->s_full[i], lead);
      return true;
    };
    for (int items = 0; ok; ++items) {
      const int nb = tp_item(x, items).nb;
      if (nb == 0) break;
      if (x.q_kept) ok = mbar_wait(&bars->q_full, items & 1, x.status, 864);
      if (ok) ok = scores(0);
      if (ok && nb > 1) ok = scores(1);
      if (ok && x.q_kept && nb <= 2) mma_commit(&bars->q_empty, lead);
      for (int b = 0; b < nb && ok; ++b) {
        const int i = b & 1;
        ok = mbar_wait(&bars->p_full[i], i ? used1 : used0, x.status, 865);
        if (i) used1 ^= 1u;
        else used0 ^= 1u;
        // the previous tile's outputs have been read
        if (ok && b == 0 && items > 0) ok = mbar_wait(&bars->o_empty, (items - 1) & 1, x.status, 866);
        if (!ok) break;
        tc_fence_after();
        const uint32_t first_acc = b > 1 ? 1u : 0u;
        if (x.v_panels == 2 && slot + 1 < x.slots) {
          // both value panels side by side: one product of 128 columns
          ok = mbar_wait(&bars->full[slot], par, x.status, 867) && mbar_wait(&bars->full[slot + 1], par, x.status, 867);
          if (!ok) break;
          tc_fence_after();
          const uint32_t bl = v_lo + slot * kStep;
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int kk = 0; kk < 8; ++kk)
              mma_ts(tm + 256 + i * 128, tm + i * 128 + (kk >> 1) * 32 + part * 16 + (kk & 1) * 8, bl + kk * 128, kIdescO2,
                     part + kk > 0 ? 1u : first_acc, lead);
          for (int vj = 0; vj < 2; ++vj) {
            mma_commit(&bars->empty[slot], lead);
            next();
          }
        } else {
          for (int vj = 0; vj < x.v_panels && ok; ++vj) {
            ok = mbar_wait(&bars->full[slot], par, x.status, 868);
            if (!ok) break;
            tc_fence_after();
            const uint32_t bl = v_lo + slot * kStep;
#pragma unroll
            for (int part = 0; part < 2; ++part)
#pragma unroll
              for (int kk = 0; kk < 8; ++kk)
                mma_ts(tm + 256 + i * 128 + vj * 64, tm + i * 128 + (kk >> 1) * 32 + part * 16 + (kk & 1) * 8, bl + kk * 128, kIdescO1,
                       part + kk > 0 ? 1u : first_acc, lead);
            mma_commit(&bars->empty[slot], lead);
            next();
          }
          if (!ok) break;
        }
        if (b + 2 < nb) {
          ok = scores(i);
          if (ok && x.q_kept && b + 3 == nb) mma_commit(&bars->q_empty, lead);
        }
        if (ok && b + 1 == nb) mma_commit(&bars->o_full, lead);
      }
    }
    __syncwarp();
  } else {
    // ------------------------------- softmax -------------------------------
    const int set = warp >> 3, half = (warp >> 2) & 1, r = (warp & 3) * 32 + lane;
    const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t ts = tmem + set * 128 + half * 64 + lanes, to = tmem + 256 + set * 128 + half * x.v_panels * 32 + lanes;
    float* peer = bars->row_max + (set * 2) * kTpTile;             // [2 halves][128]
    const float c_in = a.scale * kTpLog2e;
    const bool flip = c_in < 0.f;                                  // a negative scale: the largest score is the smallest product
    bool ok = true;
    uint32_t used = 0u;
    for (int items = 0;; ++items) {
      float m, l;
      int d1, d0, e1, e0, mine;                                    // keys d0 .. d1 of the half block are visible; e0 .. e1 to every row
      {
        const TpItem t = tp_item(x, items);
        if (t.nb == 0) break;
        // the sink counts once, in the first set
        const bool sunk = set == 0 && a.sink != nullptr;
        m = sunk ? a.sink[t.h] * kTpLog2e : -INFINITY;
        l = sunk && half == 0 ? 1.f : 0.f;
        const int k0 = t.base + (t.b0 + set) * kTpTile + half * 64;      // position of the half block's first key
        d1 = t.first + r - k0;
        d0 = talk_first(a, t.first + r) - k0;
        e1 = t.first - k0;
        e0 = talk_first(a, t.last) - k0;
        mine = t.nb > set ? (t.nb - set + 1) >> 1 : 0;             // blocks of this set
      }
      for (int n = 0; n < mine; ++n, d0 -= 2 * kTpTile, d1 -= 2 * kTpTile, e0 -= 2 * kTpTile, e1 -= 2 * kTpTile) {
        ok = ok && mbar_wait(&bars->s_full[set], used, x.status, 870);
        used ^= 1u;
        tc_fence_after();
        uint32_t s[2][32];                                         // the row's 64 scores
        tmem_ld_32x32(ts, s[0]);
        tmem_ld_32x32(ts + 32, s[1]);
        tmem_ld_wait();
        if (e1 < 63 || e0 > 0) {
#pragma unroll
          for (int j = 0; j < 64; ++j)
            if (j > d1 || j < d0) s[j >> 5][j & 31] = __float_as_uint(flip ? INFINITY : -INFINITY);
        }
        float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
        if (flip) {
#pragma unroll
          for (int j = 0; j < 64; ++j) m4[j & 3] = fmaxf(m4[j & 3], -__uint_as_float(s[j >> 5][j & 31]));
        } else {
#pragma unroll
          for (int j = 0; j < 64; ++j) m4[j & 3] = fmaxf(m4[j & 3], __uint_as_float(s[j >> 5][j & 31]));
        }
        float mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
        peer[half * kTpTile + r] = mx;
        ok = tp_bar_all(1 + set, ok);                              // the set's warps leave together
        if (!ok) break;
        mx = fmaxf(mx, peer[(half ^ 1) * kTpTile + r]) * fabsf(c_in);
        const bool grow = mx > m + 8.f || (m == -INFINITY && mx > -INFINITY);
        if (__any_sync(0xffffffffu, grow)) {
          const float f = grow ? (m == -INFINITY ? 0.f : tp_ex2(m - mx)) : 1.f;
          if (grow) m = mx;
          l *= f;
          if (n > 0) {
            // the products that fed these scores were issued after the set's previous P . V: that one is complete
            for (int c = 0; c < x.v_panels * 32; c += 8) {
              uint32_t o[8];
              tp_ld8(to + c, o);
              tmem_ld_wait();
#pragma unroll
              for (int j = 0; j < 8; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * f);
              tp_st8(to + c, o);
            }
          }
        }
        const float ms = m == -INFINITY ? 0.f : m;
        const uint64_t c2 = pack2(c_in, c_in), m2 = pack2(-ms, -ms), minus = pack2(-1.f, -1.f);
        uint64_t sum2[2] = {0ull, 0ull};
#pragma unroll
        for (int c = 0; c < 4; ++c) {                              // 16 scores: 8 columns of high parts, 8 of remainders
          uint32_t hi[8], lw[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            float p0, p1;
            unpack2(fma2(pack2(__uint_as_float(s[c >> 1][(c & 1) * 16 + 2 * j]), __uint_as_float(s[c >> 1][(c & 1) * 16 + 2 * j + 1])), c2, m2),
                    p0, p1);
            p0 = tp_ex2(p0);
            p1 = tp_ex2(p1);
            const uint64_t p2 = pack2(p0, p1);
            sum2[j & 1] = add2(sum2[j & 1], p2);
            const __nv_bfloat162 hb = __floats2bfloat162_rn(p0, p1);
            hi[j] = *reinterpret_cast<const uint32_t*>(&hb);
            float r0, r1;
            unpack2(fma2(pack2(__uint_as_float(hi[j] << 16), __uint_as_float(hi[j] & 0xffff0000u)), minus, p2), r0, r1);
            const __nv_bfloat162 lb = __floats2bfloat162_rn(r0, r1);
            lw[j] = *reinterpret_cast<const uint32_t*>(&lb);
          }
          tp_st8(ts + (c >> 1) * 32 + (c & 1) * 8, hi);
          tp_st8(ts + (c >> 1) * 32 + 16 + (c & 1) * 8, lw);
        }
        float ls[4];
        unpack2(sum2[0], ls[0], ls[1]);
        unpack2(sum2[1], ls[2], ls[3]);
        l += (ls[0] + ls[1]) + (ls[2] + ls[3]);
        tp_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&bars->p_full[set]);
      }
      // a set's denominator from its halves, then both sets' maxima and denominators meet: [set]{maximum, denominator}
      ok = tp_bar_all(1 + set, ok);
      if (half == 1) peer[kTpTile + r] = l;
      ok = tp_bar_all(1 + set, ok);
      if (half == 0) {
        l += peer[kTpTile + r];
        peer[r] = m;
        peer[kTpTile + r] = l;
      }
      ok = ok && mbar_wait(&bars->o_full, items & 1, x.status, 871);
      ok = tp_bar_all(3, ok, 512);
      tc_fence_after();
      const float m0 = bars->row_max[r], m1 = bars->row_max[2 * kTpTile + r];
      const float l0 = bars->row_max[kTpTile + r], l1 = bars->row_max[3 * kTpTile + r];
      ok = tp_bar_all(3, ok, 512);                                 // read before the next tile's maxima
      if (!ok) break;
      int again = items;
      asm volatile("" : "+r"(again));                              // formed anew: the loop above has no registers to spare
      const TpItem t = tp_item(x, again);
      const bool two = t.nb > 1;
      const float mm = fmaxf(m0, m1);
      const float f0 = m0 == -INFINITY ? 0.f : tp_ex2(m0 - mm), f1 = m1 == -INFINITY ? 0.f : tp_ex2(m1 - mm);
      const bool row_ok = r < t.n_tok;
      const long long tok = t.row0 + (row_ok ? r : 0);
      const float g = talk_gate(a, tok, t.h) / (f0 * l0 + f1 * l1);
      const float g0 = f0 * g, g1 = f1 * g;
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + tok * a.ldo;
      if (t.h == a.H - 1 && row_ok && warp < 4)
        for (int c = a.H * a.V; c < a.out_cols; ++c) out[c] = __float2bfloat16(0.f);
      out += t.h * a.V;
      const bool vec = (a.V & 7) == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0;
      const uint32_t tj = tmem + 256 + lanes;
      const int part = x.v_panels * 16, c0 = (warp >> 2) * part;   // columns of this warp: 16 or 32
      uint32_t y[4][4];                                            // results in pairs
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (e * 8 >= part) continue;
        uint32_t o[8], p[8];
        tp_ld8(tj + c0 + e * 8, o);
        if (two) tp_ld8(tj + 128 + c0 + e * 8, p);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          float u = __uint_as_float(o[2 * j]) * g0, v = __uint_as_float(o[2 * j + 1]) * g0;
          if (two) {
            u = fmaf(__uint_as_float(p[2 * j]), g1, u);
            v = fmaf(__uint_as_float(p[2 * j + 1]), g1, v);
          }
          const __nv_bfloat162 z = __floats2bfloat162_rn(u, v);
          y[e][j] = *reinterpret_cast<const uint32_t*>(&z);
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->o_empty);
      if (row_ok) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int c = c0 + e * 8;
          if (e * 8 >= part || c >= a.V) continue;
          if (vec) {
            *reinterpret_cast<uint4*>(out + c) = make_uint4(y[e][0], y[e][1], y[e][2], y[e][3]);
          } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              const __nv_bfloat162 z = *reinterpret_cast<const __nv_bfloat162*>(&y[e][j]);
              if (c + 2 * j < a.V) out[c + 2 * j] = z.x;
              if (c + 2 * j + 1 < a.V) out[c + 2 * j + 1] = z.y;
            }
          }
        }
      }
      __syncwarp();
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 17) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

struct TpShape { int k_panels, v_panels, q_kept, slots; };
static TpShape tp_shape(int G, int kp, int V) {
  TpShape s;
  s.k_panels = (G * kp + 63) / 64;
  s.v_panels = (V + 63) / 64;
  s.q_kept = s.k_panels <= kTpMaxQ ? 1 : 0;
  s.slots = (227 * 1024 - kTpBarBytes - (s.q_kept ? s.k_panels * kTpPanel : 0)) / kTpPanel;
  if (s.slots > kTpMaxSlots) s.slots = kTpMaxSlots;
  return s;
}

}  // namespace stk

using namespace stk;

// Whether the kernel covers a layer: values of at most 128 dimensions.
STK_API int stk_talking_prompt_ok(int heads, int kv_heads, int kp, int vp, int vdim) {
  return heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && kp % 16 == 0 && vp % 16 == 0 && vdim >= 1 && vdim <= 128 ? 1 : 0;
}

// rows: total rows of the gathered matrix (a multiple of 128).
STK_API int stk_talking_rows(const int* query_start, const int* req_rows, const int* start_pos, int n_req, int min_span, int chunk,
                             const int* table, int bt_stride, const void* cache, int row, void* out, long long rows, void* stream) {
  if (rows <= 0) return 0;
  if (rows % kTpTile || row % 8 || chunk < 0) return -1;
  launch_pdl(talking_rows_kernel, dim3(static_cast<unsigned>(rows / kTpTile), kTpParts), dim3(256), 0, (cudaStream_t)stream, query_start,
             req_rows, start_pos, n_req, min_span, chunk, table, bt_stride, (const __nv_bfloat16*)cache, row, (__nv_bfloat16*)out);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// Spans of at least min_span tokens.  rows [n_rows, row]: `stk_talking_rows`.
STK_API int stk_talking_prompt(const void* q, const float* gate, const float* sink, const void* rows, long long n_rows, int row,
                               int k_col, int kp, int vp, int heads, int kv_heads, int vdim, int chunk, float scale, void* out, long long ldo,
                               int out_cols, const int* query_start, const int* start_pos, int n_req, int min_span, int T, int sm_count,
                               int* status, void* stream) {
  if (T <= 0) return 0;
  TpArgs x = {};
  x.a.q = q; x.a.T = T; x.a.gate = gate; x.a.sink = sink; x.a.row = row; x.a.k_col = k_col; x.a.kp = kp; x.a.vp = vp;
  x.a.H = heads; x.a.G = kv_heads; x.a.V = vdim; x.a.chunk = chunk; x.a.scale = scale; x.a.out = out; x.a.ldo = ldo; x.a.out_cols = out_cols;
  if (!talk_ok(x.a) || !stk_talking_prompt_ok(heads, kv_heads, kp, vp, vdim) || n_req < 1 || n_rows < 1 ||
      n_rows >= (1ll << 31) || sm_count < 1 ||
      heads > 65535 || static_cast<long long>(heads) * T >= (1ll << 31) || row % 8 || row != k_col + kv_heads * kp ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(rows)) & 15))
    return -1;
  const TpShape s = tp_shape(kv_heads, kp, vdim);
  x.query_start = query_start; x.start_pos = start_pos; x.n_req = n_req; x.min_span = min_span;
  x.k_panels = s.k_panels; x.v_panels = s.v_panels; x.q_kept = s.q_kept; x.slots = s.slots; x.T = T; x.status = status;
  CUtensorMap tq, tr;
  if (make_tmap_2d(&tq, q, 2, static_cast<long long>(heads) * T, kv_heads * kp, kv_heads * kp, kTpTile) != 0) return -3;
  if (make_tmap_2d(&tr, rows, 2, n_rows, row, row, kTpTile) != 0) return -3;
  int smem = (s.q_kept ? s.k_panels * kTpPanel : 0) + s.slots * kTpPanel + kTpBarBytes;
  static_assert(sizeof(TpBars) <= kTpBarBytes, "barrier block");
  if (cudaFuncSetAttribute(talking_prompt_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -3;
  if (smem < 118 * 1024) smem = 118 * 1024;                          // one CTA per SM: it owns all of tensor memory
  const long long items = (T / kTpTile + static_cast<long long>(n_req)) * heads;       // upper bound over the ways to cut T tokens into spans
  launch_pdl(talking_prompt_tc_kernel, dim3(static_cast<unsigned>(items < sm_count ? items : sm_count)), dim3(kTpThreads), smem,
             (cudaStream_t)stream, tq, tr, x);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
