// Grouped-query sliding-window attention over paged rows, with a tanh cap on the scores and one sink logit per head.
//
// A cached row is the projected key k[0 : D] followed by the rotated copy of k[0 : R] (R = rotated dimensions): the values
// are the unrotated keys, so this one row serves as key and as value.  Scores contract over the whole row: the query is laid
// out as [0 (R columns) | q[R : D] | rot(q)[0 : R]], so a tile of rows is used in shared memory exactly as it was copied.
// Rows may also be [value (V columns) | zeros | key from column k_col on] with queries that are dense and final (rd = 0): scores
// contract the key columns and outputs sum the value columns of the same tile.  An element-wise gate and a factor can follow.
//
//   window_kv_insert       rotates the new keys and writes their rows
//   window_attn_simt       any size and type, fp32 arithmetic throughout: one CTA per (token, head)
//   window_attn_tokens     bf16, spans of a few tokens (decode): one CTA per (token, key/value head, key range); the heads of
//                          the group are the 16 MMA rows, four warps take 16 of every 64 keys each
//   window_attn_tiles      bf16, prompt portions: 128 rows (tokens x heads of the group) per CTA, key pages through two stages
// Probabilities enter the value product as bf16 pairs (high part and remainder), so they keep 16 mantissa bits.
#define STK_PDL_CLASS 8
#include "window_attention.cuh"

namespace stk {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return bf16_to_f(v); }
__device__ __forceinline__ void from_f(float* p, float v) { *p = v; }
__device__ __forceinline__ void from_f(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// cap * tanh(s / cap) through one exponential; the error is absolute, about 1e-7 of cap.
__device__ __forceinline__ float cap_score(float s, float cap, float two_over_cap) {
  const float e = __expf(s * two_over_cap);
  return cap - __fdividef(2.f * cap, 1.f + e);
}

// One warp per token; cos and sin of its position go through shared memory.  vec: rows and heads are 16-byte aligned bf16.
template <typename A>
__global__ void __launch_bounds__(128)
window_kv_insert_kernel(const WinArgs a, int T, int vec) {
  extern __shared__ float2 cs_all[];                                        // [4][rd / 2]
  pdl_wait();
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long t = blockIdx.x * 4ll + warp;
  if (t >= T) return;
  const int req = a.tok_req[t];
  const long long pos = a.positions[t];
  if (req < 0 || pos < 0) return;
  const int page = a.table[static_cast<long long>(req) * a.bt_stride + pos / kPage];
  if (page < 0) return;
  const int half = a.rd >> 1;
  float2* cs = cs_all + warp * half;
  for (int i = lane; i < half; i += 32) {
    float s, c;
    sincosf(static_cast<float>(pos) * a.freq[i], &s, &c);
    cs[i] = make_float2(c * a.mag, s * a.mag);
  }
  __syncwarp();
  const A* k = reinterpret_cast<const A*>(a.proj) + t * a.ldp + a.k_off;
  A* base = reinterpret_cast<A*>(a.cache) + (static_cast<long long>(page) * a.G * kPage + pos % kPage) * a.row;
  const long long gstep = static_cast<long long>(kPage) * a.row;
  if (sizeof(A) == 2 && vec) {
    const int c8 = a.D >> 3, h8 = half >> 3;
    for (int e = lane; e < a.G * c8; e += 32) {
      const int g = e / c8, c = (e - g * c8) * 8;
      *reinterpret_cast<uint4*>(base + g * gstep + c) = *reinterpret_cast<const uint4*>(k + g * a.D + c);
    }
    for (int e = lane; e < a.G * h8; e += 32) {
      const int g = e / h8, c = (e - g * h8) * 8;
      const uint4 uu = *reinterpret_cast<const uint4*>(k + g * a.D + c), vv = *reinterpret_cast<const uint4*>(k + g * a.D + half + c);
      uint4 ru, rv;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 u = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&uu)[i]);
        const float2 v = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&vv)[i]);
        const float2 w0 = cs[c + 2 * i], w1 = cs[c + 2 * i + 1];
        reinterpret_cast<__nv_bfloat162*>(&ru)[i] = __floats2bfloat162_rn(u.x * w0.x - v.x * w0.y, u.y * w1.x - v.y * w1.y);
        reinterpret_cast<__nv_bfloat162*>(&rv)[i] = __floats2bfloat162_rn(v.x * w0.x + u.x * w0.y, v.y * w1.x + u.y * w1.y);
      }
      A* r = base + g * gstep + a.D;
      *reinterpret_cast<uint4*>(r + c) = ru;
      *reinterpret_cast<uint4*>(r + half + c) = rv;
    }
    return;
  }
  for (int e = lane; e < a.G * a.D; e += 32) base[e / a.D * gstep + e % a.D] = k[e];
  for (int e = lane; e < a.G * half; e += 32) {
    const int g = e / half, i = e % half;
    const float u = to_f(k[g * a.D + i]), v = to_f(k[g * a.D + half + i]);
    A* r = base + g * gstep + a.D;
    from_f(r + i, u * cs[i].x - v * cs[i].y);
    from_f(r + half + i, v * cs[i].x + u * cs[i].y);
  }
}

// ---- any size, fp32 arithmetic ------------------------------------------------------------------
constexpr int kSimtKeys = 512;

template <typename A>
__global__ void __launch_bounds__(128)
window_attn_simt_kernel(const WinArgs a) {
  __shared__ float q[1024];
  __shared__ float sc[kSimtKeys];
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x, h = blockIdx.y, g = h / (a.H / a.G);
  const int req = a.tok_req[t];
  const long long pos = a.positions[t];
  A* out = reinterpret_cast<A*>(a.out) + t * a.ldo + h * a.V;
  if (req < 0 || pos < 0) {
    for (int d = threadIdx.x; d < a.V; d += blockDim.x) from_f(out + d, 0.f);
    return;
  }
  const A* qg = reinterpret_cast<const A*>(a.proj) + t * a.ldp + a.q_off + h * a.q_step;
  const int half = a.rd >> 1;
  for (int d = threadIdx.x; d < a.D; d += blockDim.x) {
    float v = to_f(qg[d]);
    if (d < a.rd) {
      const int i = d < half ? d : d - half;
      float s, c;
      sincosf(static_cast<float>(pos) * a.freq[i], &s, &c);
      const float o = to_f(qg[d < half ? d + half : d - half]);
      v = d < half ? v * (c * a.mag) - o * (s * a.mag) : v * (c * a.mag) + o * (s * a.mag);
    }
    q[d] = v;
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long lo = pos - a.window + 1 > 0 ? pos - a.window + 1 : 0;
  const int* bt = a.table + static_cast<long long>(req) * a.bt_stride;
  const A* cache = reinterpret_cast<const A*>(a.cache) + static_cast<long long>(g) * kPage * a.row;
  auto row_of = [&](long long p) {
    const int page = bt[p / kPage];
    return cache + (static_cast<long long>(page < 0 ? 0 : page) * a.G * kPage + p % kPage) * a.row;
  };
  float m = -INFINITY, l = 0.f, acc[8];
  if (a.sink != nullptr) { m = a.sink[h]; l = 1.f; }
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = 0.f;
  for (long long k0 = lo; k0 <= pos; k0 += kSimtKeys) {
    const int n = static_cast<int>(pos + 1 - k0 < kSimtKeys ? pos + 1 - k0 : kSimtKeys);
    float mx = -INFINITY;
    for (int j = warp; j < n; j += 4) {
      const A* r = row_of(k0 + j);
      float s = 0.f;
      for (int d = lane; d < a.D; d += 32) s = fmaf(q[d], to_f(d < a.rd ? r[a.D + d] : r[a.k_col - a.rd + d]), s);
      s = warp_sum(s) * a.scale;
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
      if (lane == 0) sc[j] = s;
      mx = fmaxf(mx, s);
    }
    const float m_new = fmaxf(m, block_max(mx, red));
    float sum = 0.f;
    for (int j = threadIdx.x; j < n; j += blockDim.x) {
      const float p = expf(sc[j] - m_new);
      sc[j] = p;
      sum += p;
    }
    const float f = expf(m - m_new);
    l = l * f + block_sum(sum, red);
    m = m_new;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] *= f;
    for (int j = 0; j < n; ++j) {
      const A* r = row_of(k0 + j);
      const float p = sc[j];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int d = threadIdx.x + i * 128;
        if (d < a.V) acc[i] = fmaf(p, to_f(r[d]), acc[i]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int d = threadIdx.x + i * 128;
    if (d < a.V) from_f(out + d, acc[i] / l * win_factor<A>(a, t, h, d));
  }
}

// ---- bf16 MMA building blocks -------------------------------------------------------------------
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two floats -> packed bf16 high parts and the packed bf16 remainders
__device__ __forceinline__ void split_bf16(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 r = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&r);
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// shared-memory row stride in elements: whole 16-column MMA steps plus 8 (rows fall on different banks)
__host__ __device__ inline int win_stride(int row) { return (row + 15) / 16 * 16 + 8; }

// one page of rows of key/value head g into a stage; rows outside [lo, hi] become zeros
__device__ __forceinline__ void load_page(__nv_bfloat16* stage, int stride, const WinArgs& a, const int* bt, int g,
                                          long long lp, long long lo, long long hi, int nthreads) {
  const int page = bt[lp];
  const int chunks = a.row >> 3;
  const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(a.cache) +
                             (static_cast<long long>(page < 0 ? 0 : page) * a.G + g) * kPage * a.row;
  for (int e = threadIdx.x; e < kPage * chunks; e += nthreads) {
    const int r = e / chunks, c = e - r * chunks;
    const long long p = lp * kPage + r;
    cp_async16(stage + r * stride + c * 8, src + r * a.row + c * 8, page >= 0 && p >= lo && p <= hi);
  }
}

// Query rows in the score layout.  row r of the tile: token tok(r) (index into the step, -1 none), head head(r).
template <typename TokF, typename HeadF>
__device__ __forceinline__ void fill_queries(__nv_bfloat16* qs, int stride, const WinArgs& a, int rows, int heads_per_tok,
                                             float2* cs, TokF tok, HeadF head, int nthreads) {
  const int half = a.rd >> 1;
  const int toks = (rows + heads_per_tok - 1) / heads_per_tok;
  for (int e = threadIdx.x; e < toks * half; e += nthreads) {
    const int q = e / half, i = e - q * half;
    const int t = tok(q * heads_per_tok);
    float s = 0.f, c = 0.f;
    if (t >= 0) sincosf(static_cast<float>(a.positions[t]) * a.freq[i], &s, &c);
    cs[e] = make_float2(c * a.mag, s * a.mag);
  }
  __syncthreads();
  const int cols = stride - 8;
  for (int e = threadIdx.x; e < rows * cols; e += nthreads) {
    const int r = e / cols, c = e - r * cols;
    const int t = tok(r), h = head(r);
    float v = 0.f;
    if (t >= 0 && h >= 0 && c >= a.k_col && c < a.D + a.k_col) {
      const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(a.proj) + t * a.ldp + a.q_off + h * a.q_step;
      if (a.rd == 0) {
        v = bf16_to_f(q[c - a.k_col]);
      } else if (c < a.D) {
        v = bf16_to_f(q[c]);
      } else {
        const int d = c - a.D, i = d < half ? d : d - half;
        const float2 w = cs[(r / heads_per_tok) * half + i];
        const float x = bf16_to_f(q[d]), o = bf16_to_f(q[d < half ? d + half : d - half]);
        v = d < half ? x * w.x - o * w.y : x * w.x + o * w.y;
      }
    }
    qs[r * stride + c] = __float2bfloat16(v);
  }
}

// columns between the row and the last whole MMA step are never copied: zero them once
__device__ __forceinline__ void zero_pad_columns(__nv_bfloat16* tile, int rows, int stride, int row, int nthreads) {
  const int n = stride - 8 - row;
  if (n <= 0) return;
  for (int e = threadIdx.x; e < rows * n; e += nthreads) tile[(e / n) * stride + row + e % n] = __float2bfloat16(0.f);
}

// Scores of 16 query rows against 16 keys (two n8 tiles) over the row's MMA steps [ks0, ks1).
__device__ __forceinline__ void score16(float (&s)[2][4], const __nv_bfloat16* qs, const __nv_bfloat16* keys, int stride, int ks0,
                                        int ks1, int lane) {
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
  for (int ks = ks0; ks < ks1; ++ks) {
    uint32_t af[4], bf[4];
    ldsm4(af, qs + (lane & 15) * stride + ks * 16 + (lane >> 4) * 8);
    ldsm4(bf, keys + ((lane >> 4) * 8 + (lane & 7)) * stride + ks * 16 + ((lane >> 3) & 1) * 8);
    mma16816(s[0], af, bf[0], bf[1]);
    mma16816(s[1], af, bf[2], bf[3]);
  }
}

// o += P[16 rows x 16 keys] V[16 keys x D], P as a bf16 pair
template <int NV>
__device__ __forceinline__ void value16(float (&o)[NV][4], const float (&p)[2][4], const __nv_bfloat16* keys, int stride, int D,
                                        int lane) {
  uint32_t hi[4], lo[4];
  split_bf16(p[0][0], p[0][1], hi[0], lo[0]);
  split_bf16(p[0][2], p[0][3], hi[1], lo[1]);
  split_bf16(p[1][0], p[1][1], hi[2], lo[2]);
  split_bf16(p[1][2], p[1][3], hi[3], lo[3]);
#pragma unroll
  for (int j = 0; j < NV / 2; ++j) {
    if (j * 16 < D) {
      uint32_t bf[4];
      ldsm4_t(bf, keys + ((lane & 7) + ((lane >> 3) & 1) * 8) * stride + j * 16 + (lane >> 4) * 8);
      mma16816(o[2 * j], hi, bf[0], bf[1]);
      mma16816(o[2 * j + 1], hi, bf[2], bf[3]);
      mma16816(o[2 * j], lo, bf[0], bf[1]);
      mma16816(o[2 * j + 1], lo, bf[2], bf[3]);
    }
  }
}

// ---- a few tokens per span ------------------------------------------------------------------------
// part: [splits][T][H][V + 2] fp32 (unnormalised output, maximum, denominator) when splits > 1.
template <int NV>
__global__ void __launch_bounds__(128)
window_attn_tokens_kernel(const WinArgs a, const int* __restrict__ first_pos, const int* __restrict__ last_pos, int max_span,
                          float* __restrict__ part, int T) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int stride = win_stride(a.row);
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);           // [16][stride]
  __nv_bfloat16* st = qs + 16 * stride;                                     // two stages of [64][stride]
  __shared__ float red_m[4][16], red_l[4][16];
  pdl_wait();
  pdl_trigger();
  const int splits = gridDim.x, split = blockIdx.x, t = blockIdx.z;
  const int hg = a.H / a.G, sub = (hg + 15) / 16;
  const int g = blockIdx.y / sub, h0 = g * hg + (blockIdx.y % sub) * 16;
  const int nh = min(16, (g + 1) * hg - h0);
  const int req = a.tok_req[t];
  const long long pos = a.positions[t];
  if (req < 0 || pos < 0) {
    if (split == 0)
      for (int e = threadIdx.x; e < nh * a.V; e += 128)
        reinterpret_cast<__nv_bfloat16*>(a.out)[t * a.ldo + h0 * a.V + e] = __float2bfloat16(0.f);
    return;
  }
  if (last_pos[t] - first_pos[t] + 1 > max_span) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long lo = pos - a.window + 1 > 0 ? pos - a.window + 1 : 0;
  const int* bt = a.table + static_cast<long long>(req) * a.bt_stride;
  const int p0 = static_cast<int>(lo / kPage), p1 = static_cast<int>(pos / kPage) + 1;
  const int per = (p1 - p0 + splits - 1) / splits;
  const int pa = min(p1, p0 + split * per), pb = min(p1, pa + per);
  fill_queries(qs, stride, a, 16, 16, reinterpret_cast<float2*>(st), [&](int) { return t; },
               [&](int r) { return r < nh ? h0 + r : -1; }, 128);
  __syncthreads();
  zero_pad_columns(st, 2 * kPage, stride, a.row, 128);
  const int ks0 = a.k_col / 16, ks1 = (a.D + a.k_col + 15) / 16;
  float o[NV][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int j = 0; j < NV; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[j][i] = 0.f;
  const float toc = a.softcap > 0.f ? 2.f / a.softcap : 0.f;
  if (pa < pb) load_page(st, stride, a, bt, g, pa, lo, pos, 128);
  cp_async_commit();
  for (int lp = pa; lp < pb; ++lp) {
    __nv_bfloat16* cur = st + ((lp - pa) & 1) * kPage * stride;
    if (lp + 1 < pb) load_page(st + ((lp + 1 - pa) & 1) * kPage * stride, stride, a, bt, g, lp + 1, lo, pos, 128);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const __nv_bfloat16* keys = cur + warp * 16 * stride;
    float s[2][4];
    score16(s, qs, keys, stride, ks0, ks1, lane);
    const long long kp = static_cast<long long>(lp) * kPage + warp * 16 + (lane & 3) * 2;
    float mx[2] = {m[0], m[1]};
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float v = s[i][j] * a.scale;
        if (toc > 0.f) v = cap_score(v, a.softcap, toc);
        const long long p = kp + i * 8 + (j & 1);
        if (p < lo || p > pos) v = -INFINITY;
        s[i][j] = v;
        mx[j >> 1] = fmaxf(mx[j >> 1], v);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
    }
    float f[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      f[r] = mx[r] == -INFINITY ? 1.f : __expf(m[r] - mx[r]);
      m[r] = mx[r];
      l[r] *= f[r];
    }
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float p = m[j >> 1] == -INFINITY ? 0.f : __expf(s[i][j] - m[j >> 1]);
        s[i][j] = p;
        l[j >> 1] += p;
      }
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      o[j][0] *= f[0]; o[j][1] *= f[0]; o[j][2] *= f[1]; o[j][3] *= f[1];
    }
    value16<NV>(o, s, keys, stride, a.V, lane);
    __syncthreads();
  }
  cp_async_wait<0>();
  __syncthreads();
  // merge the four warps (each saw a quarter of the keys); the output accumulators go through the stage memory
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    if ((lane & 3) == 0) {
      red_m[warp][(lane >> 2) + r * 8] = m[r];
      red_l[warp][(lane >> 2) + r * 8] = l[r];
    }
  }
  float* ob = reinterpret_cast<float*>(st);                                  // [4][16][V]
#pragma unroll
  for (int j = 0; j < NV; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = j * 8 + (lane & 3) * 2 + (i & 1), r = (lane >> 2) + (i >> 1) * 8;
      if (c < a.V) ob[(warp * 16 + r) * a.V + c] = o[j][i];
    }
  __syncthreads();
  for (int e = threadIdx.x; e < nh * a.V; e += 128) {
    const int r = e / a.V, c = e - r * a.V, h = h0 + r;
    float mm = fmaxf(fmaxf(red_m[0][r], red_m[1][r]), fmaxf(red_m[2][r], red_m[3][r]));
    if (splits == 1 && a.sink != nullptr) mm = fmaxf(mm, a.sink[h]);
    float ll = 0.f, v = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = red_m[w][r] == -INFINITY ? 0.f : __expf(red_m[w][r] - mm);
      ll = fmaf(f, red_l[w][r], ll);
      v = fmaf(f, ob[(w * 16 + r) * a.V + c], v);
    }
    if (splits == 1) {
      if (a.sink != nullptr) ll += __expf(a.sink[h] - mm);
      reinterpret_cast<__nv_bfloat16*>(a.out)[t * a.ldo + h * a.V + c] =
          __float2bfloat16(v / ll * win_factor<__nv_bfloat16>(a, t, h, c));
    } else {
      float* p = part + ((static_cast<long long>(split) * T + t) * a.H + h) * (a.V + 2);
      p[c] = v;
      if (c == 0) { p[a.V] = mm; p[a.V + 1] = ll; }
    }
  }
}

__global__ void __launch_bounds__(128)
window_attn_combine_kernel(const WinArgs a, const int* __restrict__ first_pos, const int* __restrict__ last_pos, int max_span,
                           const float* __restrict__ part, int splits, int T) {
  pdl_wait();
  pdl_trigger();
  __shared__ float s_m[64], s_w[64], s_l[64];                               // at most 64 ranges
  const int h = blockIdx.x, t = blockIdx.y;
  if (a.tok_req[t] < 0 || a.positions[t] < 0 || last_pos[t] - first_pos[t] + 1 > max_span) return;
  const long long step = static_cast<long long>(T) * a.H * (a.V + 2);
  const float* p = part + (static_cast<long long>(t) * a.H + h) * (a.V + 2);
  const int s = threadIdx.x;
  if (s < splits) {
    s_m[s] = p[s * step + a.V];
    s_l[s] = p[s * step + a.V + 1];
  }
  __syncthreads();
  float m = a.sink != nullptr ? a.sink[h] : -INFINITY;
  for (int i = 0; i < splits; ++i) m = fmaxf(m, s_m[i]);
  if (s < splits) s_w[s] = s_m[s] == -INFINITY ? 0.f : __expf(s_m[s] - m);
  __syncthreads();
  float l = a.sink != nullptr ? __expf(a.sink[h] - m) : 0.f;
  for (int i = 0; i < splits; ++i) l = fmaf(s_w[i], s_l[i], l);
  const float inv = 1.f / l;
  for (int c = s; c < a.V; c += blockDim.x) {
    float v = 0.f;
#pragma unroll 8
    for (int i = 0; i < splits; ++i) v = fmaf(s_w[i], p[i * step + c], v);
    reinterpret_cast<__nv_bfloat16*>(a.out)[t * a.ldo + h * a.V + c] =
        __float2bfloat16(v * inv * win_factor<__nv_bfloat16>(a, t, h, c));
  }
}

// ---- prompt portions --------------------------------------------------------------------------------
// WARPS x 16 rows per CTA; scores and maxima in units of log2(e).
template <int NV, int WARPS>
__global__ void __launch_bounds__(WARPS * 32, 2)
window_attn_tiles_kernel(const WinArgs a, const int* __restrict__ query_start, const int* __restrict__ req_rows,
                         const int* __restrict__ start_pos, int n_req, int min_span, int max_span, int gs) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  constexpr int kThreads = WARPS * 32, kRows = WARPS * 16;
  const int stride = win_stride(a.row);
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem_raw);           // [kRows][stride]
  __nv_bfloat16* st = qs + kRows * stride;                                  // two stages of [64][stride]
  __shared__ int s_find[2];
  pdl_wait();
  pdl_trigger();
  const int bq = kRows / gs;                                                // tokens per tile
  if (threadIdx.x == 0) {
    int left = blockIdx.x, ri = -1;
    for (int i = 0; i < n_req; ++i) {
      const int n = query_start[i + 1] - query_start[i];
      if (n < min_span || n > max_span) continue;
      const int tiles = (n + bq - 1) / bq;
      if (left < tiles) { ri = i; left = tiles - 1 - left; break; }        // the tiles with the most keys first
      left -= tiles;
    }
    s_find[0] = ri;
    s_find[1] = left;
  }
  __syncthreads();
  const int ri = s_find[0];
  if (ri < 0) return;
  const int hg = a.H / a.G, sub = (hg + gs - 1) / gs;
  const int g = blockIdx.y / sub, h0 = g * hg + (blockIdx.y % sub) * gs, h_end = min((g + 1) * hg, h0 + gs);
  const int q0 = query_start[ri], n_span = query_start[ri + 1] - q0, off = s_find[1] * bq;
  const int n_tok = min(bq, n_span - off);
  const long long first = static_cast<long long>(start_pos[ri]) + off, last = first + n_tok - 1;
  const long long lo = first - a.window + 1 > 0 ? first - a.window + 1 : 0;
  const int* bt = a.table + static_cast<long long>(req_rows[ri]) * a.bt_stride;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  auto tok_of = [&](int r) { const int q = r / gs; return q < n_tok ? q0 + off + q : -1; };
  auto head_of = [&](int r) { const int h = h0 + r % gs; return r / gs < n_tok && h < h_end ? h : -1; };
  fill_queries(qs, stride, a, kRows, gs, reinterpret_cast<float2*>(st), tok_of, head_of, kThreads);
  __syncthreads();
  zero_pad_columns(st, 2 * kPage, stride, a.row, kThreads);
  const int ks0 = a.k_col / 16, ks1 = (a.D + a.k_col + 15) / 16;
  const bool capped = a.softcap > 0.f;
  const float c_in = capped ? a.scale * 2.f * kLog2e / a.softcap : a.scale * kLog2e;
  const float c_cap = a.softcap * kLog2e, c_two = -2.f * c_cap;
  float o[NV][4], m[2], l[2] = {0.f, 0.f};
  int rel[2];                                                               // the row's token within the tile
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = warp * 16 + (lane >> 2) + r * 8;
    rel[r] = row / gs;
    const int h = head_of(row);
    m[r] = h >= 0 && a.sink != nullptr ? a.sink[h] * kLog2e : -INFINITY;
    // each of the four lanes of a row keeps a partial denominator: the sink is counted by one of them
    if (h >= 0 && a.sink != nullptr && (lane & 3) == 0) l[r] = 1.f;
  }
#pragma unroll
  for (int j = 0; j < NV; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[j][i] = 0.f;
  const int pa = static_cast<int>(lo / kPage), pb = static_cast<int>(last / kPage) + 1;
  load_page(st, stride, a, bt, g, pa, lo, last, kThreads);
  cp_async_commit();
  const __nv_bfloat16* q_frag = qs + (warp * 16 + (lane & 15)) * stride + (lane >> 4) * 8;
  for (int lp = pa; lp < pb; ++lp) {
    const __nv_bfloat16* cur = st + ((lp - pa) & 1) * kPage * stride;
    cp_async_wait<0>();
    __syncthreads();                                                        // this page is in; the other stage is free
    if (lp + 1 < pb) load_page(st + ((lp + 1 - pa) & 1) * kPage * stride, stride, a, bt, g, lp + 1, lo, last, kThreads);
    cp_async_commit();
    const long long base = static_cast<long long>(lp) * kPage;
    const bool edge = base + kPage - 1 > first || base < last - a.window + 1;
    // key position relative to the tile's first token, so that the window test is on small ints
    const int kr = static_cast<int>(base - first) + (lane & 3) * 2;
#pragma unroll 1
    for (int kh = 0; kh < kPage; kh += 32) {
      const __nv_bfloat16* keys = cur + kh * stride;
      float s[2][2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int k = 0; k < 4; ++k) s[i][j][k] = 0.f;
#pragma unroll 4
      for (int ks = ks0; ks < ks1; ++ks) {
        uint32_t af[4];
        ldsm4(af, q_frag + ks * 16);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          uint32_t bf[4];
          ldsm4(bf, keys + (i * 16 + (lane >> 4) * 8 + (lane & 7)) * stride + ks * 16 + ((lane >> 3) & 1) * 8);
          mma16816(s[i][0], af, bf[0], bf[1]);
          mma16816(s[i][1], af, bf[2], bf[3]);
        }
      }
      float mx[2] = {m[0], m[1]};
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            float v = s[i][j][k] * c_in;
            if (capped) v = fmaf(c_two, rcp(1.f + ex2(v)), c_cap);          // cap * tanh(score / cap)
            if (edge) {
              const int d = rel[k >> 1] - (kr + kh + i * 16 + j * 8 + (k & 1));   // query position - key position
              if (d < 0 || d >= a.window) v = -INFINITY;
            }
            s[i][j][k] = v;
            mx[k >> 1] = fmaxf(mx[k >> 1], v);
          }
      bool grew = false;
      float f[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        grew = grew || mx[r] > m[r];
        f[r] = mx[r] == -INFINITY ? 1.f : ex2(m[r] - mx[r]);
        m[r] = mx[r];
      }
      if (__any_sync(0xffffffffu, grew)) {                                  // most key blocks leave every maximum as it is
        l[0] *= f[0];
        l[1] *= f[1];
#pragma unroll
        for (int j = 0; j < NV; ++j) {
          o[j][0] *= f[0]; o[j][1] *= f[0]; o[j][2] *= f[1]; o[j][3] *= f[1];
        }
      }
      const float ms[2] = {m[0] == -INFINITY ? 0.f : m[0], m[1] == -INFINITY ? 0.f : m[1]};
#pragma unroll
      for (int i = 0; i < 2; ++i) {
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float p = ex2(s[i][j][k] - ms[k >> 1]);
            s[i][j][k] = p;
            l[k >> 1] += p;
          }
        value16<NV>(o, s[i], keys + i * 16 * stride, stride, a.V, lane);
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int row = warp * 16 + (lane >> 2) + r * 8;
    const int h = head_of(row);
    if (h < 0) continue;
    const float inv = 1.f / l[r];
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + tok_of(row) * a.ldo + h * a.V;
    const long long t = tok_of(row);
    const bool pair = (a.V & 1) == 0 && (a.ldo & 1) == 0;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int c = j * 8 + (lane & 3) * 2;
      float x = o[j][2 * r] * inv, y = o[j][2 * r + 1] * inv;
      if (c < a.V) x *= win_factor<__nv_bfloat16>(a, t, h, c);
      if (c + 1 < a.V) y *= win_factor<__nv_bfloat16>(a, t, h, c + 1);
      if (c + 1 < a.V && pair) {
        *reinterpret_cast<__nv_bfloat162*>(out + c) = __floats2bfloat162_rn(x, y);
      } else {
        if (c < a.V) out[c] = __float2bfloat16(x);
        if (c + 1 < a.V) out[c + 1] = __float2bfloat16(y);
      }
    }
  }
}

}  // namespace stk

using namespace stk;

#define STK_WIN_CALL proj, ldp, q_off, k_off, positions, tok_req, table, bt_stride, cache, row, freq, rd, mag, heads, kv_heads, dim

STK_API int stk_window_kv_insert(const void* proj, long long ldp, int q_off, int k_off, const int64_t* positions,
                                 const int* tok_req, const int* table, int bt_stride, void* cache, int row, const float* freq, int rd, float mag,
                                 int heads, int kv_heads, int dim,
                                 int fp32, int T, void* stream) {
  if (T <= 0) return 0;
  const WinArgs a = win_args(STK_WIN_CALL);
  if (!win_ok(a)) return -1;
  cudaStream_t st = (cudaStream_t)stream;
  const int vec = !fp32 && dim % 8 == 0 && rd % 16 == 0 && row % 8 == 0 && ldp % 8 == 0 && k_off % 8 == 0 &&
                  ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(cache)) & 15) == 0;
  const dim3 grid((T + 3) / 4);
  const size_t smem = static_cast<size_t>(2) * rd * sizeof(float2);
  if (fp32) launch_pdl(window_kv_insert_kernel<float>, grid, dim3(128), smem, st, a, T, vec);
  else launch_pdl(window_kv_insert_kernel<__nv_bfloat16>, grid, dim3(128), smem, st, a, T, vec);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_window_attention_simt(const void* proj, long long ldp, int q_off, int k_off, const int64_t* positions,
                                      const int* tok_req, const int* table, int bt_stride, void* cache, int row, const float* freq, int rd, float mag,
                                      int heads, int kv_heads, int dim,
                                      int k_col, int vdim, int q_step, const void* gate, long long ldg, float out_scale,
                                      int window, float scale, float softcap, const float* sink, void* out, long long ldo,
                                      int fp32, int T, void* stream) {
  if (T <= 0) return 0;
  WinArgs a = win_args(STK_WIN_CALL, window, scale, softcap, sink, out, ldo);
  win_layout(a, k_col, vdim, q_step, gate, ldg, out_scale);
  if (!win_ok(a) || window < 1 || heads > 65535) return -1;
  cudaStream_t st = (cudaStream_t)stream;
  if (fp32) launch_pdl(window_attn_simt_kernel<float>, dim3(T, heads), dim3(128), 0, st, a);
  else launch_pdl(window_attn_simt_kernel<__nv_bfloat16>, dim3(T, heads), dim3(128), 0, st, a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// Key ranges per (token, key/value head) so that a decode step fills the SMs, each at least two pages.
STK_API int stk_window_attention_splits(int T, int heads, int kv_heads, int window, int sm_count) {
  if (T <= 0 || kv_heads <= 0) return 1;
  const int hg = heads / kv_heads;
  const long long ctas = static_cast<long long>(T) * kv_heads * ((hg + 15) / 16);
  const int pages = (window + kPage - 1) / kPage + 1;
  long long s = (2ll * sm_count + ctas - 1) / ctas;
  if (s > (pages + 1) / 2) s = (pages + 1) / 2;
  if (s > 64) s = 64;
  return s < 1 ? 1 : static_cast<int>(s);
}

// Whether the tensor-core kernels of this file cover a layer whose rows are [value | key].
STK_API int stk_window_attention_mma_ok(int heads, int kv_heads, int dim, int vdim, int k_col, int row) {
  return heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && dim <= 256 && vdim <= 256 && k_col % 16 == 0 && row % 8 == 0 &&
         static_cast<size_t>((vdim <= 128 ? 128 : 64) + 2 * kPage) * win_stride(row) * 2 <= 220 * 1024;
}

#define STK_WIN_DIM(CALL)      \
  if (vdim <= 64) { CALL(8) }   \
  else if (vdim <= 128) { CALL(16) } \
  else { CALL(32) }

STK_API int stk_window_attention_tokens(const void* proj, long long ldp, int q_off, int k_off, const int64_t* positions,
                                        const int* tok_req, const int* table, int bt_stride, void* cache, int row, const float* freq, int rd, float mag,
                                        int heads, int kv_heads, int dim,
                                        int k_col, int vdim, int q_step, const void* gate, long long ldg, float out_scale,
                                        int window, float scale, float softcap, const float* sink, void* out, long long ldo,
                                        const int* first_pos, const int* last_pos, int max_span, int splits, float* part, int T,
                                        void* stream) {
  if (T <= 0) return 0;
  WinArgs a = win_args(STK_WIN_CALL, window, scale, softcap, sink, out, ldo);
  win_layout(a, k_col, vdim, q_step, gate, ldg, out_scale);
  if (!win_mma_ok(a) || window < 1 || splits < 1 || splits > 64 || (splits > 1 && part == nullptr) || T > 65535) return -1;
  const int sub = (heads / kv_heads + 15) / 16;
  if (kv_heads * sub > 65535) return -2;
  const size_t smem = static_cast<size_t>(16 + 2 * kPage) * win_stride(row) * 2;
  cudaStream_t st = (cudaStream_t)stream;
#define STK_WIN_TOK(NV)                                                                                                   \
  if (cudaFuncSetAttribute(window_attn_tokens_kernel<NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) !=      \
      cudaSuccess)                                                                                                         \
    return -3;                                                                                                             \
  launch_pdl(window_attn_tokens_kernel<NV>, dim3(splits, kv_heads * sub, T), dim3(128), smem, st, a, first_pos, last_pos,  \
             max_span, part, T);
  STK_WIN_DIM(STK_WIN_TOK)
#undef STK_WIN_TOK
  if (splits > 1)
    launch_pdl(window_attn_combine_kernel, dim3(heads, T), dim3(128), 0, st, a, first_pos, last_pos, max_span, part, splits, T);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_window_attention_tiles(const void* proj, long long ldp, int q_off, int k_off, const int64_t* positions,
                                       const int* tok_req, const int* table, int bt_stride, void* cache, int row, const float* freq, int rd, float mag,
                                       int heads, int kv_heads, int dim,
                                       int k_col, int vdim, int q_step, const void* gate, long long ldg, float out_scale,
                                       int window, float scale, float softcap, const float* sink, void* out, long long ldo,
                                       const int* query_start, const int* req_rows, const int* start_pos, int n_req, int min_span, int max_span,
                                       int T, void* stream) {
  if (T <= 0) return 0;
  WinArgs a = win_args(STK_WIN_CALL, window, scale, softcap, sink, out, ldo);
  win_layout(a, k_col, vdim, q_step, gate, ldg, out_scale);
  if (!win_mma_ok(a) || window < 1 || n_req < 1) return -1;
  // eight warps of rows up to 128-wide heads, four above (their output accumulators fill the register file)
  const int rows = vdim <= 128 ? 128 : 64;
  const int hg = heads / kv_heads, gs = hg < rows ? hg : rows, sub = (hg + gs - 1) / gs, bq = rows / gs;
  if (kv_heads * sub > 65535) return -2;
  const size_t smem = static_cast<size_t>(rows + 2 * kPage) * win_stride(row) * 2;
  const dim3 grid(T / bq + n_req, kv_heads * sub);                     // upper bound over the ways to cut T tokens into spans
  cudaStream_t st = (cudaStream_t)stream;
#define STK_WIN_TILE(NV)                                                                                                  \
  {                                                                                                                       \
    constexpr int kW = NV <= 16 ? 8 : 4;                                                                                   \
    if (cudaFuncSetAttribute(window_attn_tiles_kernel<NV, kW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) !=  \
        cudaSuccess)                                                                                                       \
      return -3;                                                                                                           \
    launch_pdl(window_attn_tiles_kernel<NV, kW>, grid, dim3(kW * 32), smem, st, a, query_start, req_rows, start_pos, n_req, \
               min_span, max_span, gs);                                                                                              \
  }
  STK_WIN_DIM(STK_WIN_TILE)
#undef STK_WIN_TILE
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
