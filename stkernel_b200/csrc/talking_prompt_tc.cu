// Talking-heads attention of prompt portions on the 5th-generation tensor cores (bf16).  Mixed queries meet the keys of all key/value heads
// side by side, so a head's scores contract kv_heads * kp columns; its values are those of its own key/value head.
//
//   talking_rows         the cached rows that a request's long span can see, copied out of their pages into one matrix; each request
//                        starts on a 128-row border and is padded with zero rows to the next one
//   talking_prompt_tc    one CTA per (tile of 128 query tokens, head) over blocks of 128 keys
//
//     loader warp      the tile's queries (kept in shared memory; where they are too wide, a panel at a time with the keys) and, through a
//                      ring of 16 KB panels [128 rows x 64 columns], keys and values in the order in which they are used
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

constexpr int kTpTile = 128, kTpPanel = kTpTile * 128, kTpThreads = 576, kTpMaxSlots = 12, kTpMaxQ = 10;
constexpr float kTpLog2e = 1.4426950408889634f;

struct alignas(8) TpBars {
  uint64_t q_full, full[kTpMaxSlots], empty[kTpMaxSlots];
  uint64_t s_full[2], p_full[2], o_full[2];
  uint32_t tmem_base;
  int find[2];
  long long seg;
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

__device__ __forceinline__ void tp_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
      "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
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
  float* row_sum = reinterpret_cast<float*>(ring);                 // [set][half][row], when nothing uses the ring any more
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_trigger();
  if (threadIdx.x == 0) {
    int left = blockIdx.x, ri = -1;
    long long seg = 0;
    for (int i = 0; i < x.n_req; ++i) {
      const int n = x.query_start[i + 1] - x.query_start[i];
      if (n < x.min_span) continue;
      const int tiles = (n + kTpTile - 1) / kTpTile;
      if (left < tiles) { ri = i; left = tiles - 1 - left; break; }      // the longest contexts of a request first
      left -= tiles;
      seg += (x.start_pos[i] + n - tp_base(a.chunk, x.start_pos[i]) + kTpTile - 1) / kTpTile * kTpTile;
    }
    bars->find[0] = ri;
    bars->find[1] = left;
    bars->seg = seg;
    mbar_init(&bars->q_full, 1);
    for (int s = 0; s < kTpMaxSlots; ++s) {
      mbar_init(&bars->full[s], 1);
      mbar_init(&bars->empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->s_full[i], 1);
      mbar_init(&bars->p_full[i], 8);
      mbar_init(&bars->o_full[i], 1);
    }
    fence_barrier_init();
  }
  __syncthreads();
  const int ri = bars->find[0];
  if (ri < 0) return;
  if (warp == 17) {
    tmem_alloc(&bars->tmem_base, 512);
    tmem_relinquish();
  }
  const int h = blockIdx.y;
  const int q0 = x.query_start[ri], span = x.query_start[ri + 1] - q0, off = bars->find[1] * kTpTile;
  const int n_tok = min(kTpTile, span - off), first = x.start_pos[ri] + off, last = first + n_tok - 1;
  const int base = tp_base(a.chunk, x.start_pos[ri]), seg = static_cast<int>(bars->seg);
  const int b0 = (talk_first(a, first) - base) / kTpTile, nb = (last - base) / kTpTile + 1 - b0;      // blocks of gathered rows
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_base;                           // scores of set i: i * 128; outputs: 256 + i * 128

  if (warp == 16) {
    // ------------------------------- loader -------------------------------
    if (lane == 0) {
      bool ok = true;
      int seq = 0;
      if (x.q_kept) {
        mbar_expect_tx(&bars->q_full, kp * kTpPanel);
        for (int p = 0; p < kp; ++p) tma_load_2d(q_s + p * kTpPanel, &tm_q, &bars->q_full, p * 64, h * x.T + q0 + off);
      }
      auto load = [&](const CUtensorMap* tm, int col, int y) {
        const int st = seq % x.slots;
        if (seq >= x.slots) ok = mbar_wait(&bars->empty[st], ((seq / x.slots) - 1) & 1, x.status, 860);
        if (!ok) return;
        mbar_expect_tx(&bars->full[st], kTpPanel);
        tma_load_2d(ring + st * kTpPanel, tm, &bars->full[st], col, y);
        ++seq;
      };
      auto keys = [&](int b) {
        for (int j = 0; j < kp && ok; ++j) {
          if (!x.q_kept) load(&tm_q, j * 64, h * x.T + q0 + off);
          if (ok) load(&tm_r, a.k_col + j * 64, seg + (b0 + b) * kTpTile);
        }
      };
      const int vc = h / (a.H / a.G) * a.vp;
      keys(0);
      if (nb > 1) keys(1);
      for (int b = 0; b < nb && ok; ++b) {
        for (int j = 0; j < x.v_panels && ok; ++j) load(&tm_r, vc + j * 64, seg + (b0 + b) * kTpTile);
        if (b + 2 < nb) keys(b + 2);
      }
      if (!ok) {
        // leave no copy in flight: what was asked for lands before the CTA's shared memory goes away
        if (x.q_kept) mbar_wait(&bars->q_full, 0, nullptr, 0);
        for (int s = max(0, seq - x.slots); s < seq; ++s) mbar_wait(&bars->full[s % x.slots], (s / x.slots) & 1, nullptr, 0);
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
    uint32_t par = 0u;
    auto next = [&]() {
      if (++slot == x.slots) { slot = 0; par ^= 1u; }
    };
    bool ok = !x.q_kept || mbar_wait(&bars->q_full, 0, x.status, 861);
    auto scores = [&](int b) {
      const int i = b & 1;
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
    if (ok) ok = scores(0);
    if (ok && nb > 1) ok = scores(1);
    for (int b = 0; b < nb && ok; ++b) {
      const int i = b & 1;
      ok = mbar_wait(&bars->p_full[i], (b >> 1) & 1, x.status, 864);
      if (!ok) break;
      tc_fence_after();
      const uint32_t first_acc = b > 1 ? 1u : 0u;
      if (x.v_panels == 2 && slot + 1 < x.slots) {
        // both value panels side by side: one product of 128 columns
        ok = mbar_wait(&bars->full[slot], par, x.status, 865) && mbar_wait(&bars->full[slot + 1], par, x.status, 865);
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
          ok = mbar_wait(&bars->full[slot], par, x.status, 866);
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
      if (b + 2 >= nb) mma_commit(&bars->o_full[i], lead);
      else ok = scores(b + 2);
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
    const uint32_t masked = __float_as_uint(flip ? INFINITY : -INFINITY);
    // the sink counts once, in the first set
    const bool sunk = set == 0 && a.sink != nullptr;
    float m = sunk ? a.sink[h] * kTpLog2e : -INFINITY, l = sunk && half == 0 ? 1.f : 0.f;
    const int pos = first + r, lo = talk_first(a, pos), lo_last = talk_first(a, last);
    const int mine = nb > set ? (nb - set + 1) >> 1 : 0;           // blocks of this set
    bool ok = true;
    for (int n = 0; n < mine; ++n) {
      const int k0 = base + (b0 + 2 * n + set) * kTpTile + half * 64;      // position of the half block's first key
      ok = ok && mbar_wait(&bars->s_full[set], n & 1, x.status, 870);
      tc_fence_after();
      const int d1 = pos - k0, d0 = lo - k0;                       // keys d0 .. d1 of the half block are visible
      uint32_t s[2][32];                                           // the row's 64 scores
      tmem_ld_32x32(ts, s[0]);
      tmem_ld_32x32(ts + 32, s[1]);
      tmem_ld_wait();
      if (k0 + 63 > first || k0 < lo_last) {
#pragma unroll
        for (int j = 0; j < 64; ++j)
          if (j > d1 || j < d0) s[j >> 5][j & 31] = masked;
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
      ok = tp_bar_all(1 + set, ok);                                // the set's warps leave together
      if (!ok) break;
      mx = fmaxf(mx, peer[(half ^ 1) * kTpTile + r]) * fabsf(c_in);
      const bool grow = mx > m + 8.f || (m == -INFINITY && mx > -INFINITY);
      if (__any_sync(0xffffffffu, grow)) {
        const float f = grow ? (m == -INFINITY ? 0.f : tp_ex2(m - mx)) : 1.f;
        if (grow) m = mx;
        l *= f;
        if (n > 0) {
          // the products that fed these scores were issued after the set's previous P . V: that one is complete
          for (int c = 0; c < x.v_panels * 32; c += 16) {
            uint32_t o[16];
            tmem_ld_32x16(to + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * f);
            tp_st16(to + c, o);
          }
        }
      }
      const float ms = m == -INFINITY ? 0.f : m;
      const uint64_t c2 = pack2(c_in, c_in), m2 = pack2(-ms, -ms), minus = pack2(-1.f, -1.f);
      uint64_t sum2[2] = {0ull, 0ull};
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        uint32_t hi[16], lw[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          float p0, p1;
          unpack2(fma2(pack2(__uint_as_float(s[c][2 * j]), __uint_as_float(s[c][2 * j + 1])), c2, m2), p0, p1);
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
        tp_st16(ts + c * 32, hi);
        tp_st16(ts + c * 32 + 16, lw);
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
    // both outputs complete: their maxima and denominators meet, and each warp writes a quarter of the columns
    if (ok) ok = mbar_wait(&bars->o_full[0], 0, x.status, 871) && (nb < 2 || mbar_wait(&bars->o_full[1], 0, x.status, 872));
    if (half == 0) bars->row_max[set * 2 * kTpTile + r] = m;
    row_sum[(set * 2 + half) * kTpTile + r] = l;
    tc_fence_before();
    ok = tp_bar_all(3, ok, 512);
    tc_fence_after();
    if (ok) {
      const bool two = nb > 1;
      const float m0 = bars->row_max[r], m1 = bars->row_max[2 * kTpTile + r];
      const float l0 = row_sum[r] + row_sum[kTpTile + r], l1 = row_sum[2 * kTpTile + r] + row_sum[3 * kTpTile + r];
      const float mm = fmaxf(m0, m1);
      const float f0 = m0 == -INFINITY ? 0.f : tp_ex2(m0 - mm), f1 = m1 == -INFINITY ? 0.f : tp_ex2(m1 - mm);
      const bool row_ok = r < n_tok;
      const long long t = q0 + off + (row_ok ? r : 0);
      const float g = talk_gate(a, t, h) / (f0 * l0 + f1 * l1);
      const float g0 = f0 * g, g1 = f1 * g;
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + t * a.ldo;
      if (h == a.H - 1 && row_ok && warp < 4)
        for (int c = a.H * a.V; c < a.out_cols; ++c) out[c] = __float2bfloat16(0.f);
      out += h * a.V;
      const bool vec = (a.V & 7) == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0;
      const uint32_t tj = tmem + 256 + lanes;
      const int part = x.v_panels * 16;                            // columns of this warp
      for (int c = (warp >> 2) * part; c < ((warp >> 2) + 1) * part; c += 16) {
        uint32_t o[16], p[16];
        __syncwarp();
        tmem_ld_32x16(tj + c, o);
        if (two) tmem_ld_32x16(tj + 128 + c, p);
        tmem_ld_wait();
        if (!row_ok) continue;
        float y[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          y[j] = __uint_as_float(o[j]) * g0;
          if (two) y[j] = fmaf(__uint_as_float(p[j]), g1, y[j]);
        }
        if (vec) {
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            if (c + q * 8 >= a.V) continue;
            uint32_t pk[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              const __nv_bfloat162 v = __floats2bfloat162_rn(y[q * 8 + 2 * j], y[q * 8 + 2 * j + 1]);
              pk[j] = *reinterpret_cast<const uint32_t*>(&v);
            }
            *reinterpret_cast<uint4*>(out + c + q * 8) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
          }
        } else {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (c + j < a.V) out[c + j] = __float2bfloat16(y[j]);
        }
      }
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
                               int out_cols, const int* query_start, const int* start_pos, int n_req, int min_span, int T, int* status,
                               void* stream) {
  if (T <= 0) return 0;
  TpArgs x = {};
  x.a.q = q; x.a.T = T; x.a.gate = gate; x.a.sink = sink; x.a.row = row; x.a.k_col = k_col; x.a.kp = kp; x.a.vp = vp;
  x.a.H = heads; x.a.G = kv_heads; x.a.V = vdim; x.a.chunk = chunk; x.a.scale = scale; x.a.out = out; x.a.ldo = ldo; x.a.out_cols = out_cols;
  if (!talk_ok(x.a) || !stk_talking_prompt_ok(heads, kv_heads, kp, vp, vdim) || n_req < 1 || n_rows < 1 || n_rows >= (1ll << 31) ||
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
  launch_pdl(talking_prompt_tc_kernel, dim3(T / kTpTile + n_req, heads), dim3(kTpThreads), smem, (cudaStream_t)stream, tq, tr, x);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
