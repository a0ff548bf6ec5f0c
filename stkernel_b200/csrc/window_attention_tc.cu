// Sliding-window attention of prompt portions on the 5th-generation tensor cores (bf16, head size a multiple of 16 up to 128).
//
// One CTA takes two tiles of 128 query rows (tokens x heads of a group) over the key pages both need:
//
//   loader warp      brings pages of 64 rows in by TMA as panels of [64 rows x 64 columns], 128-byte swizzled, through a ring;
//                    rows outside the CTA's key range are zeroed on the way
//   MMA warp         S[row, key] = Q . K^T per tile (both K-major), and O[row, dim] += P . V with the same page as MN-major
//                    operand: a cached row is key and value at once.  While one tile's softmax runs, the other tile's
//                    products do.
//   softmax warps    four per tile, one row per thread: scores from TMEM, tanh cap, window, running maximum (O is rescaled in
//                    TMEM only when a row's maximum grew by more than 2^8), probabilities to shared memory as bf16 pairs
//                    (high part and remainder, two products), row output from TMEM
//
// TMEM: per tile two buffers of 64 score columns (the next page's scores are ready when a softmax warp comes back for them)
// and up to 128 columns of O.  Every mbarrier wait is bounded; on expiry the status word is set and the CTA leaves.  Layout of the query rows: see window_attention.cu.
#define STK_PDL_CLASS 8
#include "window_attention.cuh"

namespace stk {

int make_tmap_2d(CUtensorMap* tm, const void* base, int elem_bytes, long long rows, long long cols, long long ld, int box_rows);

constexpr int kTcTileRows = 128, kTcThreads = 320, kTcMaxStages = 4;
constexpr int kTcKvPanel = kPage * 128, kTcQPanel = kTcTileRows * 128, kTcPTile = kTcTileRows * 128;

struct alignas(8) WinTcBars {
  uint64_t loaded[kTcMaxStages], full[kTcMaxStages], empty[kTcMaxStages];
  uint64_t s_full[2][2], p_full[2], pv_done[2];             // [tile][score buffer], [tile]
  uint32_t tmem_base;
  int find[2];
};

struct WinTcArgs {
  WinArgs w;
  const int* query_start; const int* req_rows; const int* start_pos;
  int n_req, min_span, gs;
  int panels, q_panel0, q_panels, stages;
  int* status;
};

__device__ __forceinline__ void win_tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
      "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
// MN-major operand, 128-byte swizzle: 64-column blocks are `lbo` bytes apart along N, 8-row groups 1024 bytes along K.
__device__ __forceinline__ uint64_t win_desc_mn(uint32_t smem_addr, uint32_t lbo) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>(lbo >> 4) << 16;
  d |= static_cast<uint64_t>(1024 >> 4) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}

template <bool kCap>
__global__ void __launch_bounds__(kTcThreads, 1)
window_attn_tc_kernel(const __grid_constant__ CUtensorMap tm_kv, const WinTcArgs x) {
  extern __shared__ uint8_t smem_raw[];
  const WinArgs& a = x.w;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_s = smem;                                             // [2 tiles][q_panels][128 rows x 128 B]
  uint8_t* p_s = q_s + 2 * x.q_panels * kTcQPanel;                 // [2 tiles]{high, remainder}[128 rows x 128 B]
  uint8_t* kv_s = p_s + 4 * kTcPTile;                              // [stages][panels][64 rows x 128 B]
  WinTcBars* bars = reinterpret_cast<WinTcBars*>(kv_s + x.stages * x.panels * kTcKvPanel);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_wait();
  pdl_trigger();
  const int bq = kTcTileRows / x.gs;                               // tokens per tile
  if (threadIdx.x == 0) {
    int left = blockIdx.x, ri = -1;
    for (int i = 0; i < x.n_req; ++i) {
      const int n = x.query_start[i + 1] - x.query_start[i];
      if (n < x.min_span) continue;
      const int tiles = (n + 2 * bq - 1) / (2 * bq);
      if (left < tiles) { ri = i; left = tiles - 1 - left; break; }
      left -= tiles;
    }
    bars->find[0] = ri;
    bars->find[1] = left;
    for (int s = 0; s < kTcMaxStages; ++s) {
      mbar_init(&bars->loaded[s], 1);
      mbar_init(&bars->full[s], 1);
      mbar_init(&bars->empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->s_full[i][0], 1);
      mbar_init(&bars->s_full[i][1], 1);
      mbar_init(&bars->p_full[i], 4);
      mbar_init(&bars->pv_done[i], 1);
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
  const int hg = a.H / a.G, sub = (hg + x.gs - 1) / x.gs;
  const int g = blockIdx.y / sub, h0 = g * hg + (blockIdx.y % sub) * x.gs, h_end = min((g + 1) * hg, h0 + x.gs);
  const int q0 = x.query_start[ri], span = x.query_start[ri + 1] - q0, off = bars->find[1] * 2 * bq;
  const long long pos0 = x.start_pos[ri];
  const int* bt = a.table + static_cast<long long>(x.req_rows[ri]) * a.bt_stride;
  // per tile: tokens, first position and pages [pa, pb)
  int n_tok[2], pa[2], pb[2];
  long long first[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    n_tok[i] = max(0, min(bq, span - off - i * bq));
    first[i] = pos0 + off + i * bq;
    const long long lo = first[i] - a.window + 1 > 0 ? first[i] - a.window + 1 : 0;
    pa[i] = static_cast<int>(lo / kPage);
    pb[i] = n_tok[i] > 0 ? static_cast<int>((first[i] + n_tok[i] - 1) / kPage) + 1 : pa[i];
  }
  const int page0 = pa[0], page1 = max(pb[0], pb[1]);              // tile 0 always has tokens
  const long long key_lo = first[0] - a.window + 1 > 0 ? first[0] - a.window + 1 : 0;
  const long long key_hi = pos0 + min(span, off + 2 * bq) - 1;

  // ---- query rows: [zeros below R | q[R : D] | rotated q[0 : R]], K-major panels --------------------------------------
  {
    const int half = a.rd >> 1;
    float2* cs = reinterpret_cast<float2*>(p_s);                   // [2 * bq][half], the probabilities come later
    for (int e = threadIdx.x; e < 2 * bq * half; e += kTcThreads) {
      const int q = e / half, i = e - q * half;
      float s = 0.f, c = 0.f;
      if (off + q < span) sincosf(static_cast<float>(pos0 + off + q) * a.freq[i], &s, &c);
      cs[e] = make_float2(c * a.mag, s * a.mag);
    }
    __syncthreads();
    const int ch = x.q_panels * 8;
    for (int e = threadIdx.x; e < 2 * kTcTileRows * ch; e += kTcThreads) {
      const int rr = e / ch, cc = e - rr * ch;                     // row over both tiles, 16-byte chunk
      const int tile = rr >> 7, r = rr & 127, q = r / x.gs, h = h0 + (r - q * x.gs);
      const bool ok = q < n_tok[tile] && h < h_end && q < bq;
      const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(a.proj) +
                                 (ok ? static_cast<long long>(q0 + off + tile * bq + q) * a.ldp + a.q_off + h * a.D : 0);
      __nv_bfloat16 v[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int c = x.q_panel0 * 64 + cc * 8 + i;
        float f = 0.f;
        if (ok && c >= a.rd && c < a.D + a.rd) {
          if (c < a.D) {
            f = bf16_to_f(src[c]);
          } else {
            const int d = c - a.D, k = d < half ? d : d - half;
            const float2 w = cs[(tile * bq + q) * half + k];
            const float u = bf16_to_f(src[d]), o = bf16_to_f(src[d < half ? d + half : d - half]);
            f = d < half ? u * w.x - o * w.y : u * w.x + o * w.y;
          }
        }
        v[i] = __float2bfloat16(f);
      }
      uint8_t* dst = q_s + (tile * x.q_panels + (cc >> 3)) * kTcQPanel + r * 128 + (((cc & 7) ^ (r & 7)) << 4);
      *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(v);
    }
  }
  fence_proxy_async();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_base;                           // scores of tile i, buffer b: i * 64 + b * 128; outputs: 256 + i * 128

  if (warp == 8) {
    // ------------------------------- loader -------------------------------
    // A page is complete before the next one is asked for, so that a page never waits behind the release of a stage that only
    // a later product gives back; the ring still runs stages ahead of the products.
    bool ok = true;
    const int n = page1 - page0;
    for (int i = 0; i < n && ok; ++i) {
      const int st = i % x.stages;
      if (i >= x.stages) ok = mbar_wait(&bars->empty[st], ((i / x.stages) - 1) & 1, x.status, 700);
      if (!ok) break;
      if (lane == 0) {
        const int page = max(bt[page0 + i], 0);
        mbar_expect_tx(&bars->loaded[st], x.panels * kTcKvPanel);
        for (int p = 0; p < x.panels; ++p)
          tma_load_2d(kv_s + (st * x.panels + p) * kTcKvPanel, &tm_kv, &bars->loaded[st], p * 64, (page * a.G + g) * kPage);
      }
      __syncwarp();
      ok = mbar_wait(&bars->loaded[st], (i / x.stages) & 1, x.status, 701);
      if (!ok) break;
      const long long base = static_cast<long long>(page0 + i) * kPage;
      if (base < key_lo || base + kPage - 1 > key_hi) {
        for (int e = lane; e < kPage * x.panels * 8; e += 32) {
          const int r = e / (x.panels * 8), c = e - r * (x.panels * 8);
          if (base + r < key_lo || base + r > key_hi)
            *reinterpret_cast<uint4*>(kv_s + (st * x.panels + (c >> 3)) * kTcKvPanel + r * 128 + ((c & 7) << 4)) =
                make_uint4(0, 0, 0, 0);
        }
        fence_proxy_async();
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->full[st]);
    }
    if (!ok && lane == 0) {
      // leave no copy in flight: the ring's outstanding loads land before the CTA's shared memory goes away
      for (int s = 0; s < x.stages; ++s) {
        mbar_wait(&bars->loaded[s], 0, nullptr, 0);
        mbar_wait(&bars->loaded[s], 1, nullptr, 0);
      }
    }
  } else if (warp == 9) {
    // ------------------------------- MMA issuer -------------------------------
    if (lane == 0) {
      const uint32_t idesc_qk = umma_idesc(1u, 1u, 128, kPage);
      const uint32_t idesc_pv = umma_idesc(1u, 1u, 128, a.D) | (1u << 16);        // B is MN-major
      const int ks0 = a.rd / 16, ks1 = (a.D + a.rd + 15) / 16;
      int done[2] = {0, 0};
      bool ok = true;
      // pages that the scores run ahead of the outputs; page lp + lead must fit the ring beside page lp
      const int lead = x.stages > 2 ? 2 : 1;
      for (int lp = page0 - lead; lp < page1 && ok; ++lp) {
        const int n = lp - page0, st = n % x.stages, sn = (n + lead) % x.stages;
        bool waited = false;
        for (int i = 0; i < 2 && ok; ++i) {
          const bool now = lp >= pa[i] && lp < pb[i], next = lp + lead >= pa[i] && lp + lead < pb[i];
          if (now) {
            ok = mbar_wait(&bars->p_full[i], done[i] & 1, x.status, 710 + i);
            if (!ok) break;
            tc_fence_after();
          }
          if (next) {
            if (!waited) {
              ok = mbar_wait(&bars->full[sn], ((n + lead) / x.stages) & 1, x.status, 712);
              if (!ok) break;
              tc_fence_after();
              waited = true;
            }
            const uint8_t* kv = kv_s + sn * x.panels * kTcKvPanel;
            const int buf = (lp + lead - pa[i]) & 1;
            for (int ks = ks0; ks < ks1; ++ks) {
              const uint64_t ad = umma_desc_sw128(smem_u32(q_s + (i * x.q_panels + (ks >> 2) - x.q_panel0) * kTcQPanel)) + 2 * (ks & 3);
              const uint64_t bd = umma_desc_sw128(smem_u32(kv + (ks >> 2) * kTcKvPanel)) + 2 * (ks & 3);
              umma_f16(tmem + i * 64 + buf * 128, ad, bd, idesc_qk, ks > ks0 ? 1u : 0u);
            }
            umma_commit(&bars->s_full[i][buf]);
          }
          if (now) {
            const uint8_t* kv = kv_s + st * x.panels * kTcKvPanel;
#pragma unroll
            for (int part = 0; part < 2; ++part)
#pragma unroll
              for (int kk = 0; kk < 4; ++kk) {
                const uint64_t ad = umma_desc_sw128(smem_u32(p_s + (2 * i + part) * kTcPTile)) + 2 * kk;
                const uint64_t bd = win_desc_mn(smem_u32(kv + kk * 2048), kTcKvPanel);
                umma_f16(tmem + 256 + i * 128, ad, bd, idesc_pv, (done[i] > 0 || part > 0 || kk > 0) ? 1u : 0u);
              }
            umma_commit(&bars->pv_done[i]);
            ++done[i];
          }
        }
        if (ok && n >= 0) umma_commit(&bars->empty[st]);
      }
    }
    __syncwarp();
  } else {
    // ------------------------------- softmax -------------------------------
    const int tile = warp >> 2, r = (warp & 3) * 32 + lane;
    const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t ts = tmem + tile * 64 + lanes, to = tmem + 256 + tile * 128 + lanes;
    const int q = r / x.gs, h = h0 + (r - q * x.gs);
    const bool row_ok = q < n_tok[tile] && q < bq && h < h_end;
    const float c_in = kCap ? a.scale * 2.f * kLog2e / a.softcap : a.scale * kLog2e;
    const float c_cap = a.softcap * kLog2e, c_two = -2.f * c_cap;
    float m = row_ok && a.sink != nullptr ? a.sink[h] * kLog2e : -INFINITY, l = row_ok && a.sink != nullptr ? 1.f : 0.f;
    const long long last = first[tile] + n_tok[tile] - 1;
    uint8_t* p_hi = p_s + 2 * tile * kTcPTile + r * 128;
    uint8_t* p_lo = p_hi + kTcPTile;
    bool ok = true;
    int k = 0;
    for (int lp = pa[tile]; lp < pb[tile] && ok; ++lp, ++k) {
      ok = mbar_wait(&bars->s_full[tile][k & 1], (k >> 1) & 1, x.status, 720);
      if (!ok) break;
      tc_fence_after();
      float v[64];
      {
        uint32_t s0[32], s1[32];
        tmem_ld_32x32(ts + (k & 1) * 128, s0);
        tmem_ld_32x32(ts + (k & 1) * 128 + 32, s1);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          v[j] = __uint_as_float(s0[j]);
          v[32 + j] = __uint_as_float(s1[j]);
        }
      }
      const long long base = static_cast<long long>(lp) * kPage;
      const bool edge = base + kPage - 1 > first[tile] || base < last - a.window + 1;
      const int d0 = static_cast<int>(first[tile] + q - base);              // query position - key position of column 0
      // cap * tanh(score / cap), in units of log2(e)
#pragma unroll
      for (int j = 0; j < 64; ++j) {
        const float u = v[j] * c_in;
        v[j] = kCap ? fmaf(c_two, rcp(1.f + ex2(u)), c_cap) : u;
      }
      if (edge) {
#pragma unroll
        for (int j = 0; j < 64; ++j)
          if (d0 - j < 0 || d0 - j >= a.window) v[j] = -INFINITY;
      }
      float mx4[4] = {v[0], v[1], v[2], v[3]};
#pragma unroll
      for (int j = 4; j < 64; ++j) mx4[j & 3] = fmaxf(mx4[j & 3], v[j]);
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      const bool grow = mx > m + 8.f || (m == -INFINITY && mx > -INFINITY);
      const bool any = __any_sync(0xffffffffu, grow);
      if (k > 0) {
        // the previous product has read this tile's probabilities and finished its output
        ok = mbar_wait(&bars->pv_done[tile], (k - 1) & 1, x.status, 721);
        if (!ok) break;
        tc_fence_after();
      }
      if (any) {
        const float f = grow && m != -INFINITY ? ex2(m - mx) : (grow ? 0.f : 1.f);
        if (grow) m = mx;
        l *= f;
        if (k > 0) {
          for (int c = 0; c < a.D; c += 16) {
            uint32_t o[16];
            tmem_ld_32x16(to + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 16; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * f);
            win_tmem_st16(to + c, o);
          }
          asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
        }
      }
      const float ms = m == -INFINITY ? 0.f : m;
      float ls[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float p0 = ex2(v[c * 8 + 2 * j] - ms), p1 = ex2(v[c * 8 + 2 * j + 1] - ms);
          ls[j] += p0 + p1;
          const __nv_bfloat162 hb = __floats2bfloat162_rn(p0, p1);
          const float2 hf = __bfloat1622float2(hb);
          const __nv_bfloat162 lb = __floats2bfloat162_rn(p0 - hf.x, p1 - hf.y);
          hi[j] = *reinterpret_cast<const uint32_t*>(&hb);
          lo[j] = *reinterpret_cast<const uint32_t*>(&lb);
        }
        const int at = (c ^ (r & 7)) << 4;
        *reinterpret_cast<uint4*>(p_hi + at) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(p_lo + at) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
      l += (ls[0] + ls[1]) + (ls[2] + ls[3]);
      fence_proxy_async();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->p_full[tile]);
    }
    if (ok && k > 0) ok = mbar_wait(&bars->pv_done[tile], (k - 1) & 1, x.status, 722);
    tc_fence_after();
    if (ok && k > 0) {
      const float inv = 1.f / l;
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + static_cast<long long>(q0 + off + tile * bq + q) * a.ldo + h * a.D;
      for (int c = 0; c < a.D; c += 16) {
        uint32_t o[16];
        tmem_ld_32x16(to + c, o);
        tmem_ld_wait();
        if (row_ok) {
          uint32_t pk[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            const __nv_bfloat162 b = __floats2bfloat162_rn(__uint_as_float(o[2 * j]) * inv, __uint_as_float(o[2 * j + 1]) * inv);
            pk[j] = *reinterpret_cast<const uint32_t*>(&b);
          }
          *reinterpret_cast<uint4*>(out + c) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
          *reinterpret_cast<uint4*>(out + c + 8) = make_uint4(pk[4], pk[5], pk[6], pk[7]);
        }
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

}  // namespace stk

using namespace stk;
// Whether the kernel covers a layer: bf16 rows of whole 16-byte units, head size a multiple of 16 up to 128.
STK_API int stk_window_attention_tc_ok(int heads, int kv_heads, int dim, int rd, int row) {
  return heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim % 16 == 0 && dim <= 128 && rd % 2 == 0 && rd <= dim &&
         row % 8 == 0 && row >= dim + rd && row <= 256;
}

// Spans of at least min_span tokens.
STK_API int stk_window_attention_tc(const void* proj, long long ldp, int q_off, int k_off, const int64_t* positions,
                                    const int* tok_req, const int* table, int bt_stride, void* cache, int row, const float* freq, int rd,
                                    float mag, int heads, int kv_heads, int dim, int window, float scale, float softcap,
                                    const float* sink, void* out, long long ldo, const int* query_start, const int* req_rows,
                                    const int* start_pos, int n_req, int min_span, long long num_pages, int T, int* status, void* stream) {
  if (T <= 0) return 0;
  WinTcArgs x;
  x.w = win_args(proj, ldp, q_off, k_off, positions, tok_req, table, bt_stride, cache, row, freq, rd, mag, heads, kv_heads, dim,
                 window, scale, softcap, sink, out, ldo);
  if (!stk_window_attention_tc_ok(heads, kv_heads, dim, rd, row) || window < 1 || n_req < 1 || num_pages < 1 || ldo % 8 ||
      ((reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(cache)) & 15))
    return -1;
  x.query_start = query_start; x.req_rows = req_rows; x.start_pos = start_pos;
  x.n_req = n_req; x.min_span = min_span; x.status = status;
  const int hg = heads / kv_heads;
  x.gs = hg < kTcTileRows ? hg : kTcTileRows;
  const int sub = (hg + x.gs - 1) / x.gs, bq = kTcTileRows / x.gs;
  if (kv_heads * sub > 65535) return -2;
  x.panels = (dim + rd + 63) / 64;
  x.q_panel0 = rd / 16 / 4;
  x.q_panels = x.panels - x.q_panel0;
  const int fixed = 2 * x.q_panels * kTcQPanel + 4 * kTcPTile + 512 + 1024;
  x.stages = (227 * 1024 - fixed) / (x.panels * kTcKvPanel);
  if (x.stages > kTcMaxStages) x.stages = kTcMaxStages;
  if (x.stages < 2) return -5;
  static_assert(sizeof(WinTcBars) <= 512, "barrier block");
  int smem = fixed + x.stages * x.panels * kTcKvPanel;
  if (smem < 118 * 1024) smem = 118 * 1024;                          // one CTA per SM: it owns all of tensor memory
  CUtensorMap tm;
  if (make_tmap_2d(&tm, cache, 2, num_pages * kv_heads * kPage, row, row, kPage) != 0) return -3;
  if (cudaFuncSetAttribute(window_attn_tc_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess ||
      cudaFuncSetAttribute(window_attn_tc_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess)
    return -3;
  const dim3 grid(T / (2 * bq) + n_req, kv_heads * sub);
  if (softcap > 0.f) launch_pdl(window_attn_tc_kernel<true>, grid, dim3(kTcThreads), smem, (cudaStream_t)stream, tm, x);
  else launch_pdl(window_attn_tc_kernel<false>, grid, dim3(kTcThreads), smem, (cudaStream_t)stream, tm, x);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
