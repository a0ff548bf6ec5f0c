// Causal attention of prompt portions over the full context on the 5th-generation tensor cores (bf16).  Latent attention: keys and
// values of the whole context are expanded from the cached latents first (a plain product), then each head is ordinary causal
// attention.  Grouped attention: the gathered rows themselves hold the keys and values of every key/value head.
//
//   latent_rows          the cached rows of every request with a long span, copied out of their pages into one matrix; each
//                        request starts on a 128-row border and is padded with zero rows to the next one
//   latent_prompt_tc     one CTA per (two tiles of 128 query tokens, head) over blocks of 128 keys
//
//     loader warp      query tiles and, through a ring of 16 KB panels [128 rows x 64 columns], per block the head's expanded
//                      keys, the rotated key part (shared by all heads, straight from the rows) and the expanded values
//     MMA warp         S[query, key] = Q . K^T per tile, then O[query, v] += P . V with P read from tensor memory; the two tiles
//                      alternate, so one tile's softmax runs under the other's products
//     softmax warps    four per tile, one row per thread: running maximum (O rescaled only when a row's maximum grew by more
//                      than 2^8), probabilities written over the scores as bf16 pairs (high part and remainder, two products)
//
// TMEM: per tile 128 columns of scores / probabilities and up to 128 of O.  A 32-column chunk of scores is replaced by 16 columns of
// packed high parts and 16 of remainders of the same keys.  Every mbarrier wait is bounded.
#define STK_PDL_CLASS 8
#include "latent_attention.cuh"

namespace stk {

int make_tmap_2d(CUtensorMap* tm, const void* base, int elem_bytes, long long rows, long long cols, long long ld, int box_rows);

constexpr int kLpTile = 128, kLpPanel = kLpTile * 128, kLpThreads = 320, kLpMaxSlots = 12;
constexpr float kLpLog2e = 1.4426950408889634f;

struct alignas(8) LpBars {
  uint64_t q_full, full[kLpMaxSlots], empty[kLpMaxSlots];
  uint64_t s_full[2], p_full[2], o_full[2];
  uint32_t tmem_base;
  int find[2];
  long long seg;
};

struct LpArgs {
  const __nv_bfloat16* qr; long long ldqr;             // rotated query parts before rotation: head h at columns h * R
  const float* gate; long long ldg;
  const int* query_start; const int* start_pos;
  int n_req, min_span;
  const float* freq;
  int R, rot_off;
  int h0;                                              // first head of this launch
  int dp, d_panels, r_panels, v_panels, d_steps;       // panels of 64 columns; d_steps: 16-column steps of the unrotated part
  float scale;
  __nv_bfloat16* out; long long ldo; int vp, vdim;     // head h's output at columns h * vp; vw columns of it are written
  int vw;
  int h0_kv, heads_per_kv, kv_step, k_off, v_off;      // keys of a head at columns (h - h0_kv) / heads_per_kv * kv_step + k_off
  const float* sink;                                   // per head: score of a key without value (nullptr: none)
  const __nv_bfloat16* ogate; long long ldog;          // element-wise output gate logits, head h at columns h * vp (nullptr: none)
  float out_scale;
  int slots;
  int* status;
};

__device__ __forceinline__ void lp_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
      "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ void lp_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ float lp_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// kRowParts CTAs per 128 rows of the gathered matrix.
constexpr int kRowParts = 8;
__global__ void __launch_bounds__(256)
latent_rows_kernel(const int* __restrict__ query_start, const int* __restrict__ req_rows, const int* __restrict__ start_pos, int n_req,
                   int min_span, const int* __restrict__ table, int bt_stride, const __nv_bfloat16* __restrict__ cache, int G, int row,
                   __nv_bfloat16* __restrict__ out) {
  __shared__ int found[3];
  pdl_wait();
  pdl_trigger();
  if (threadIdx.x == 0) {
    int left = blockIdx.x, ri = -1, ctx = 0;
    for (int i = 0; i < n_req; ++i) {
      const int n = query_start[i + 1] - query_start[i];
      if (n < min_span) continue;
      ctx = start_pos[i] + n;
      const int tiles = (ctx + kLpTile - 1) / kLpTile;
      if (left < tiles) { ri = i; break; }
      left -= tiles;
    }
    found[0] = ri; found[1] = left; found[2] = ctx;
  }
  __syncthreads();
  const int ri = found[0], j0 = found[1] * kLpTile, ctx = found[2];
  const int per_head = row >> 3, chunks = G * per_head;            // a page is [G][kLatPage][row], an output row [G * row]
  constexpr int kRows = kLpTile / kRowParts;
  const int part = blockIdx.y * kRows;
  uint4* dst = reinterpret_cast<uint4*>(out + (static_cast<long long>(blockIdx.x) * kLpTile + part) * G * row);
  const int* bt = ri >= 0 ? table + static_cast<long long>(req_rows[ri]) * bt_stride : nullptr;
  for (int e = threadIdx.x; e < kRows * chunks; e += blockDim.x) {
    const int r = e / chunks, ce = e - r * chunks, g = ce / per_head, c = ce - g * per_head, j = j0 + part + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (ri >= 0 && j < ctx) {
      const int page = bt[j / kLatPage];
      if (page >= 0)
        v = *reinterpret_cast<const uint4*>(cache + ((static_cast<long long>(page) * G + g) * kLatPage + j % kLatPage) * row + c * 8);
    }
    dst[e] = v;
  }
}

__global__ void __launch_bounds__(kLpThreads, 1)
latent_prompt_tc_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_e,
                        const __grid_constant__ CUtensorMap tm_r, const LpArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int kp = a.d_panels + a.r_panels, per = kp + a.v_panels;
  uint8_t* q_s = smem;                                             // [2 tiles][kp][128 rows x 128 B]
  uint8_t* ring = q_s + 2 * kp * kLpPanel;                         // [slots][128 rows x 128 B]
  LpBars* bars = reinterpret_cast<LpBars*>(ring + a.slots * kLpPanel);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_trigger();
  if (threadIdx.x == 0) {
    int left = blockIdx.x, ri = -1;
    long long seg = 0;
    for (int i = 0; i < a.n_req; ++i) {
      const int n = a.query_start[i + 1] - a.query_start[i];
      if (n < a.min_span) continue;
      const int tiles = (n + 2 * kLpTile - 1) / (2 * kLpTile);
      if (left < tiles) { ri = i; left = tiles - 1 - left; break; }      // the longest contexts of a request first
      left -= tiles;
      seg += (a.start_pos[i] + n + kLpTile - 1) / kLpTile * kLpTile;
    }
    bars->find[0] = ri;
    bars->find[1] = left;
    bars->seg = seg;
    mbar_init(&bars->q_full, 1);
    for (int s = 0; s < kLpMaxSlots; ++s) {
      mbar_init(&bars->full[s], 1);
      mbar_init(&bars->empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->s_full[i], 1);
      mbar_init(&bars->p_full[i], 4);
      mbar_init(&bars->o_full[i], 1);
    }
    fence_barrier_init();
  }
  __syncthreads();
  const int ri = bars->find[0];
  if (ri < 0) return;
  if (warp == 9) {
    tmem_alloc(&bars->tmem_base, 512);
    tmem_relinquish();
  }
  const int hl = blockIdx.y, h = a.h0 + hl;
  const int q0 = a.query_start[ri], span = a.query_start[ri + 1] - q0, off = bars->find[1] * 2 * kLpTile;
  const int pos0 = a.start_pos[ri];
  const int seg = static_cast<int>(bars->seg);
  int n_tok[2], first[2], nb[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    n_tok[i] = max(0, min(kLpTile, span - off - i * kLpTile));
    first[i] = pos0 + off + i * kLpTile;
    nb[i] = n_tok[i] > 0 ? (first[i] + n_tok[i] + kLpTile - 1) / kLpTile : 0;
  }
  const int nb_max = max(nb[0], nb[1]);

  if (warp == 8 && lane == 0) {
    mbar_expect_tx(&bars->q_full, 2 * a.d_panels * kLpPanel);
    for (int i = 0; i < 2; ++i)
      for (int p = 0; p < a.d_panels; ++p)
        tma_load_2d(q_s + (i * kp + p) * kLpPanel, &tm_q, &bars->q_full, h * a.dp + p * 64, q0 + off + i * kLpTile);
  }
  // rotated query part: pairs of columns, zeros behind the last one
  {
    const int pairs = a.R >> 1, cols = a.r_panels * 32;
    for (int e = threadIdx.x; e < 2 * kLpTile * cols; e += kLpThreads) {
      const int rr = e / cols, c = e - rr * cols;                  // row over both tiles, pair
      const int i = rr >> 7, r = rr & 127;
      uint32_t v = 0;
      if (c < pairs && r < (i ? n_tok[1] : n_tok[0])) {
        const __nv_bfloat16* src = a.qr + static_cast<long long>(q0 + off + rr) * a.ldqr + h * a.R + 2 * c;
        const float2 w = cos_sin_split((i ? first[1] : first[0]) + r, a.freq[c], a.freq[pairs + c]);
        const float x = bf16_to_f(src[0]), y = bf16_to_f(src[1]);
        const __nv_bfloat162 b = __floats2bfloat162_rn(x * w.x - y * w.y, y * w.x + x * w.y);
        v = *reinterpret_cast<const uint32_t*>(&b);
      }
      uint8_t* dst = q_s + (i * kp + a.d_panels + (c >> 5)) * kLpPanel + r * 128 + ((((c & 31) >> 2) ^ (r & 7)) << 4) + (c & 3) * 4;
      *reinterpret_cast<uint32_t*>(dst) = v;
    }
  }
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_base;                           // scores of tile i: i * 128; outputs: 256 + i * 128

  if (warp == 8) {
    // ------------------------------- loader -------------------------------
    if (lane == 0) {
      bool ok = true;
      int seq = 0;
      for (int b = 0; b < nb_max && ok; ++b) {
        for (int j = 0; j < per; ++j, ++seq) {
          const int st = seq % a.slots;
          if (seq >= a.slots) ok = mbar_wait(&bars->empty[st], ((seq / a.slots) - 1) & 1, a.status, 800);
          if (!ok) break;
          mbar_expect_tx(&bars->full[st], kLpPanel);
          const int y = seg + b * kLpTile;
          const int e0 = (h - a.h0_kv) / a.heads_per_kv * a.kv_step;
          if (j < a.d_panels) tma_load_2d(ring + st * kLpPanel, &tm_e, &bars->full[st], e0 + a.k_off + j * 64, y);
          else if (j < kp) tma_load_2d(ring + st * kLpPanel, &tm_r, &bars->full[st], a.rot_off + (j - a.d_panels) * 64, y);
          else tma_load_2d(ring + st * kLpPanel, &tm_e, &bars->full[st], e0 + a.v_off + (j - kp) * 64, y);
        }
      }
      if (!ok) {
        // leave no copy in flight: what was asked for lands before the CTA's shared memory goes away
        for (int k = max(0, seq - a.slots); k < seq; ++k)
          mbar_wait(&bars->full[k % a.slots], (k / a.slots) & 1, nullptr, 0);
      }
    }
    __syncwarp();
  } else if (warp == 9) {
    // ------------------------------- MMA issuer -------------------------------
    const uint32_t lead = elect_one() ? 1u : 0u, tm = __shfl_sync(0xffffffffu, tmem, 0);
    constexpr uint32_t kIdescS = umma_idesc(1u, 1u, 128, 128);
    constexpr uint32_t kIdescO1 = umma_idesc(1u, 1u, 128, 64) | (1u << 16), kIdescO2 = umma_idesc(1u, 1u, 128, 128) | (1u << 16);
    constexpr uint32_t kStep = kLpPanel >> 4;                      // a panel in descriptor units
    const uint32_t q_lo = desc_lo(smem_u32(q_s)), k_lo = desc_lo(smem_u32(ring)), v_lo = desc_lo(smem_u32(ring), kLpPanel);
    bool ok = mbar_wait(&bars->q_full, 0, a.status, 810);
    struct At { int slot; uint32_t par; };
    auto ahead = [&](At c, int n) {
      c.slot += n;
      if (c.slot >= a.slots) { c.slot -= a.slots; c.par ^= 1u; }
      return c;
    };
    At cur{0, 0u};                                                 // first panel of block b
    auto scores = [&](int i, At c, bool wait) {
      for (int j = 0; j < kp; ++j) {
        const At p = ahead(c, j);
        if (wait) {
          if (!mbar_wait(&bars->full[p.slot], p.par, a.status, 811)) return false;
          tc_fence_after();
        }
        const uint32_t al = q_lo + (i * kp + j) * kStep, bl = k_lo + p.slot * kStep;
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) mma_ss(tm + i * 128, al + 2 * ks, bl + 2 * ks, kIdescS, ks > 0 ? 1u : (j > 0 ? 1u : 0u), lead);
      }
      mma_commit(&bars->s_full[i], lead);
      return true;
    };
    if (ok) ok = scores(0, cur, true);
    if (ok && nb[1] > 0) ok = scores(1, cur, false);
    if (ok)
      for (int j = 0; j < kp; ++j) mma_commit(&bars->empty[j], lead);
    for (int b = 0; b < nb_max && ok; ++b) {
      const At next = ahead(cur, per), v0 = ahead(cur, kp);
      bool v_seen = false, k_seen = false;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        if (!ok || b >= nb[i]) continue;
        ok = mbar_wait(&bars->p_full[i], b & 1, a.status, 812);
        tc_fence_after();
        if (ok && !v_seen) {
          for (int j = 0; j < a.v_panels && ok; ++j) {
            const At p = ahead(v0, j);
            ok = mbar_wait(&bars->full[p.slot], p.par, a.status, 813);
          }
          tc_fence_after();
          v_seen = true;
        }
        if (!ok) continue;
        const uint32_t first_acc = b > 0 ? 1u : 0u;
        if (a.v_panels == 2 && v0.slot + 1 < a.slots) {
          // both value panels side by side: one product of 128 columns
          const uint32_t bl = v_lo + v0.slot * kStep;
#pragma unroll
          for (int part = 0; part < 2; ++part)
#pragma unroll
            for (int kk = 0; kk < 8; ++kk)
              mma_ts(tm + 256 + i * 128, tm + i * 128 + (kk >> 1) * 32 + part * 16 + (kk & 1) * 8, bl + kk * 128, kIdescO2,
                     part + kk > 0 ? 1u : first_acc, lead);
        } else {
          for (int vj = 0; vj < a.v_panels; ++vj) {
            const uint32_t bl = v_lo + ahead(v0, vj).slot * kStep;
#pragma unroll
            for (int part = 0; part < 2; ++part)
#pragma unroll
              for (int kk = 0; kk < 8; ++kk)
                mma_ts(tm + 256 + i * 128 + vj * 64, tm + i * 128 + (kk >> 1) * 32 + part * 16 + (kk & 1) * 8, bl + kk * 128,
                       kIdescO1, part + kk > 0 ? 1u : first_acc, lead);
          }
        }
        if (b + 1 == nb[i]) {
          mma_commit(&bars->o_full[i], lead);
        } else {
          ok = scores(i, next, !k_seen);
          k_seen = true;
        }
      }
      if (ok) {
        for (int j = 0; j < a.v_panels; ++j) mma_commit(&bars->empty[ahead(v0, j).slot], lead);
        if (b + 1 < nb_max)
          for (int j = 0; j < kp; ++j) mma_commit(&bars->empty[ahead(next, j).slot], lead);
      }
      cur = next;
    }
    __syncwarp();
  } else {
    // ------------------------------- softmax -------------------------------
    const int tile = warp >> 2, r = (warp & 3) * 32 + lane;
    const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t ts = tmem + tile * 128 + lanes, to = tmem + 256 + tile * 128 + lanes;
    const int t_first = tile ? first[1] : first[0], t_blocks = tile ? nb[1] : nb[0], t_tok = tile ? n_tok[1] : n_tok[0];
    const float c_in = a.scale * kLpLog2e;
    const bool flip = c_in < 0.f;                                  // a negative scale: the largest score is the smallest product
    const uint32_t masked = __float_as_uint(flip ? INFINITY : -INFINITY);
    float m = a.sink != nullptr ? a.sink[h] * kLpLog2e : -INFINITY, l = a.sink != nullptr ? 1.f : 0.f;
    bool ok = true;
    for (int b = 0; b < t_blocks && ok; ++b) {
      ok = mbar_wait(&bars->s_full[tile], b & 1, a.status, 820);
      if (!ok) break;
      tc_fence_after();
      const int d0 = t_first + r - b * kLpTile;                    // keys 0 .. d0 of the block are visible
      const bool edge = b * kLpTile + kLpTile - 1 > t_first;
      uint32_t s[2][32];                                           // 64 scores of the row at a time
      auto fetch = [&](int half) {
        tmem_ld_32x32(ts + half * 64, s[0]);
        tmem_ld_32x32(ts + half * 64 + 32, s[1]);
        tmem_ld_wait();
        if (edge) {
#pragma unroll
          for (int j = 0; j < 64; ++j)
            if (half * 64 + j > d0) s[j >> 5][j & 31] = masked;
        }
      };
      auto largest = [&]() {
        float m4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < 64; ++j) {
          const float v = __uint_as_float(s[j >> 5][j & 31]);
          m4[j & 3] = fmaxf(m4[j & 3], flip ? -v : v);
        }
        return fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
      };
      fetch(0);
      float mx = largest();
      fetch(1);
      mx = fmaxf(mx, largest()) * fabsf(c_in);
      const bool grow = mx > m + 8.f || (m == -INFINITY && mx > -INFINITY);
      if (__any_sync(0xffffffffu, grow)) {
        const float f = grow ? (m == -INFINITY ? 0.f : lp_ex2(m - mx)) : 1.f;
        if (grow) m = mx;
        l *= f;
        if (b > 0) {
          // the products that fed these scores were issued after the previous P . V: that one is complete
          for (int c = 0; c < a.v_panels * 64; c += 16) {
            uint32_t o[16];
            tmem_ld_32x16(to + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * f);
            lp_st16(to + c, o);
          }
          lp_st_wait();
        }
      }
      const float ms = m == -INFINITY ? 0.f : m;
      const uint64_t c2 = pack2(c_in, c_in), m2 = pack2(-ms, -ms), minus = pack2(-1.f, -1.f);
      uint64_t sum2[2] = {0ull, 0ull};
      auto weigh = [&](int half) {
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          uint32_t hi[16], lo[16];
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            float p0, p1;
            unpack2(fma2(pack2(__uint_as_float(s[c][2 * j]), __uint_as_float(s[c][2 * j + 1])), c2, m2), p0, p1);
            p0 = lp_ex2(p0);
            p1 = lp_ex2(p1);
            const uint64_t p2 = pack2(p0, p1);
            sum2[j & 1] = add2(sum2[j & 1], p2);
            const __nv_bfloat162 hb = __floats2bfloat162_rn(p0, p1);
            hi[j] = *reinterpret_cast<const uint32_t*>(&hb);
            float r0, r1;
            unpack2(fma2(pack2(__uint_as_float(hi[j] << 16), __uint_as_float(hi[j] & 0xffff0000u)), minus, p2), r0, r1);
            const __nv_bfloat162 lb = __floats2bfloat162_rn(r0, r1);
            lo[j] = *reinterpret_cast<const uint32_t*>(&lb);
          }
          lp_st16(ts + (half * 2 + c) * 32, hi);
          lp_st16(ts + (half * 2 + c) * 32 + 16, lo);
        }
      };
      weigh(1);
      fetch(0);
      weigh(0);
      float ls[4];
      unpack2(sum2[0], ls[0], ls[1]);
      unpack2(sum2[1], ls[2], ls[3]);
      l += (ls[0] + ls[1]) + (ls[2] + ls[3]);
      lp_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->p_full[tile]);
    }
    if (ok && t_blocks > 0) {
      ok = mbar_wait(&bars->o_full[tile], 0, a.status, 821);
      tc_fence_after();
      if (ok) {
        const bool row_ok = r < t_tok;
        const long long t = q0 + off + tile * kLpTile + (row_ok ? r : 0);
        const float g = (a.gate != nullptr ? lat_sigmoid(a.gate[t * a.ldg + h]) : 1.f) * a.out_scale / l;
        __nv_bfloat16* out = a.out + t * a.ldo + h * a.vp;
        const __nv_bfloat16* og = a.ogate != nullptr ? a.ogate + t * a.ldog + h * a.vp : nullptr;
        const bool vec = ((a.vp | a.vw) & 7) == 0 && ((reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(og)) & 15) == 0;
        for (int c = 0; c < a.v_panels * 64; c += 16) {
          uint32_t o[16];
          __syncwarp();
          tmem_ld_32x16(to + c, o);
          tmem_ld_wait();
          if (!row_ok) continue;
          if (vec) {
#pragma unroll
            for (int half = 0; half < 2; ++half) {
              if (c + half * 8 >= a.vw) continue;
              uint4 gv = make_uint4(0, 0, 0, 0);
              if (og != nullptr) gv = *reinterpret_cast<const uint4*>(og + c + half * 8);
              uint32_t pk[4];
#pragma unroll
              for (int j = 0; j < 4; ++j) {
                float x = __uint_as_float(o[half * 8 + 2 * j]) * g, y = __uint_as_float(o[half * 8 + 2 * j + 1]) * g;
                if (og != nullptr) {
                  const float2 z = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&gv)[j]);
                  x = __fdividef(x, 1.f + __expf(-z.x));
                  y = __fdividef(y, 1.f + __expf(-z.y));
                }
                const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
                pk[j] = *reinterpret_cast<const uint32_t*>(&v);
              }
              *reinterpret_cast<uint4*>(out + c + half * 8) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
            }
          } else {
#pragma unroll
            for (int j = 0; j < 16; ++j)
              if (c + j < a.vw) {
                float x = __uint_as_float(o[j]) * g;
                if (og != nullptr) x *= lat_sigmoid(bf16_to_f(og[c + j]));
                out[c + j] = __float2bfloat16(x);
              }
          }
        }
        if (row_ok)
          for (int c = a.v_panels * 64; c < a.vw; c += 8) *reinterpret_cast<uint4*>(out + c) = make_uint4(0, 0, 0, 0);
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

static int lp_slots(int dp, int rot, int vdim) {
  const int kp = dp / 64 + (rot + 63) / 64;
  const int s = (225 * 1024 - 2 * kp * kLpPanel) / kLpPanel;
  return s > kLpMaxSlots ? kLpMaxSlots : s;
}

}  // namespace stk

using namespace stk;

// Whether the kernel covers a layer: values of at most 128 dimensions, and a ring that holds a block's keys and values.
STK_API int stk_latent_prompt_ok(int dim, int dp, int rot, int vdim, int row, int rot_off) {
  if (dim < 1 || dp % 64 || dp < dim || rot < 0 || (rot & 1) || vdim < 1 || vdim > 128 || row % 8 || rot_off % 8) return 0;
  const int per = dp / 64 + (rot + 63) / 64 + (vdim + 63) / 64;
  return lp_slots(dp, rot, vdim) >= per;
}

// rows: total rows of the gathered matrix (a multiple of 128).  Pages hold `heads` blocks of [64, row]; a gathered row is theirs
// side by side.
STK_API int stk_latent_rows(const int* query_start, const int* req_rows, const int* start_pos, int n_req, int min_span,
                            const int* table, int bt_stride, const void* cache, int heads, int row, void* out, long long rows,
                            void* stream) {
  if (rows <= 0) return 0;
  if (rows % kLpTile || row % 8 || heads < 1) return -1;
  launch_pdl(latent_rows_kernel, dim3(static_cast<unsigned>(rows / kLpTile), kRowParts), dim3(256), 0, (cudaStream_t)stream, query_start,
             req_rows, start_pos, n_req, min_span, table, bt_stride, (const __nv_bfloat16*)cache, heads, row, (__nv_bfloat16*)out);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// Spans of at least min_span tokens, heads [h0, h0 + nh).  q: unrotated query parts of all heads (head h at columns h * dp);
// rows: gathered cached rows; kv [rows, nh * (dp + v64)]: their expansion, per head keys then values (v64: vdim rounded up to 64).
STK_API int stk_latent_prompt(const void* q, long long ldq, const void* qr, long long ldqr, const float* gate, long long ldg,
                              const int* query_start, const int* start_pos, int n_req, int min_span, const void* rows,
                              long long n_rows, int row, int rot_off, const void* kv, const float* freq, int heads, int h0, int nh,
                              int dim, int dp, int rot, int vdim, int vp, float scale, void* out, long long ldo, int T, int* status,
                              void* stream) {
  if (T <= 0 || nh <= 0) return 0;
  if (!stk_latent_prompt_ok(dim, dp, rot, vdim, row, rot_off) || n_req < 1 || n_rows < 1 || h0 < 0 || h0 + nh > heads || nh > 65535 ||
      ldo % 8 || ldq % 8 || vp % 8 || vp < (vdim + 63) / 64 * 64 || n_rows >= (1ll << 31) ||
      ((reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv)) & 15))
    return -1;
  LpArgs a;
  a.qr = (const __nv_bfloat16*)qr; a.ldqr = ldqr; a.gate = gate; a.ldg = ldg;
  a.query_start = query_start; a.start_pos = start_pos; a.n_req = n_req; a.min_span = min_span;
  a.freq = freq; a.R = rot; a.rot_off = rot_off; a.h0 = h0;
  a.dp = dp; a.d_panels = dp / 64; a.r_panels = (rot + 63) / 64; a.v_panels = (vdim + 63) / 64; a.d_steps = (dim + 15) / 16;
  a.scale = scale; a.out = (__nv_bfloat16*)out; a.ldo = ldo; a.vp = vp; a.vdim = vdim; a.vw = vp; a.status = status;
  a.h0_kv = h0; a.heads_per_kv = 1; a.kv_step = dp + a.v_panels * 64; a.k_off = 0; a.v_off = dp;
  a.sink = nullptr; a.ogate = nullptr; a.ldog = 0; a.out_scale = 1.f;
  a.slots = lp_slots(dp, rot, vdim);
  CUtensorMap tq, te, tr;
  const long long cols = static_cast<long long>(nh) * (dp + a.v_panels * 64);
  if (make_tmap_2d(&tq, q, 2, T, static_cast<long long>(heads) * dp, ldq, kLpTile) != 0) return -3;
  if (make_tmap_2d(&te, kv, 2, n_rows, cols, cols, kLpTile) != 0) return -3;
  if (make_tmap_2d(&tr, rows, 2, n_rows, row, row, kLpTile) != 0) return -3;
  const int smem = 2 * (a.d_panels + a.r_panels) * kLpPanel + a.slots * kLpPanel + 1024 + 1024;
  static_assert(sizeof(LpBars) <= 1024, "barrier block");
  if (cudaFuncSetAttribute(latent_prompt_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess)
    return -3;
  // at least 118 KB: one CTA per SM, it owns all of tensor memory
  launch_pdl(latent_prompt_tc_kernel, dim3(T / (2 * kLpTile) + n_req, nh), dim3(kLpThreads), smem < 118 * 1024 ? 118 * 1024 : smem,
             (cudaStream_t)stream, tq, te, tr, a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// Whether `stk_prompt_attention` covers a layer: values of at most 128 dimensions, a ring that holds a block's keys and values.
STK_API int stk_prompt_attention_ok(int dim, int dp, int vdim, int row, int k_col) {
  if (row % 8 || k_col % 8 || k_col < vdim || row < k_col + dim) return 0;
  return stk_latent_prompt_ok(dim, dp, 0, vdim, row, 0);
}

// Spans of at least min_span tokens.  q: final queries, head h at columns h * dp (zeros behind dim); rows [n_rows, kv_heads * row]:
// gathered cached rows, per key/value head value, then key from column k_col on.  out: head h at columns h * vdim.
STK_API int stk_prompt_attention(const void* q, long long ldq, const int* query_start, const int* start_pos, int n_req, int min_span,
                                 const void* rows, long long n_rows, int row, int k_col, const void* gate, long long ldg, float out_scale,
                                 const float* sink, int heads, int kv_heads, int dim, int dp, int vdim, float scale, void* out,
                                 long long ldo, int T, int* status, void* stream) {
  if (T <= 0) return 0;
  if (!stk_prompt_attention_ok(dim, dp, vdim, row, k_col) || n_req < 1 || n_rows < 1 || heads < 1 || heads > 65535 || kv_heads < 1 ||
      heads % kv_heads || ldq % 8 || n_rows >= (1ll << 31) || ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(rows)) & 15))
    return -1;
  LpArgs a = {};
  a.query_start = query_start; a.start_pos = start_pos; a.n_req = n_req; a.min_span = min_span;
  a.dp = dp; a.d_panels = dp / 64; a.r_panels = 0; a.v_panels = (vdim + 63) / 64; a.d_steps = (dim + 15) / 16;
  a.scale = scale; a.out = (__nv_bfloat16*)out; a.ldo = ldo; a.vp = vdim; a.vdim = vdim; a.vw = vdim; a.status = status;
  a.h0_kv = 0; a.heads_per_kv = heads / kv_heads; a.kv_step = row; a.k_off = k_col; a.v_off = 0;
  a.sink = sink; a.ogate = (const __nv_bfloat16*)gate; a.ldog = ldg; a.out_scale = out_scale;
  a.slots = lp_slots(dp, 0, vdim);
  CUtensorMap tq, te;
  const long long cols = static_cast<long long>(kv_heads) * row;
  if (make_tmap_2d(&tq, q, 2, T, static_cast<long long>(heads) * dp, ldq, kLpTile) != 0) return -3;
  if (make_tmap_2d(&te, rows, 2, n_rows, cols, cols, kLpTile) != 0) return -3;
  const int smem = 2 * a.d_panels * kLpPanel + a.slots * kLpPanel + 1024 + 1024;
  if (cudaFuncSetAttribute(latent_prompt_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess)
    return -3;
  launch_pdl(latent_prompt_tc_kernel, dim3(T / (2 * kLpTile) + n_req, heads), dim3(kLpThreads), smem < 118 * 1024 ? 118 * 1024 : smem,
             (cudaStream_t)stream, tq, te, te, a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
