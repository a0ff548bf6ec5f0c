// Time mixing: a linear recurrence with a decay per head and key channel that the token chooses, read out before its update with a bonus
// for the current token (ops/recurrence.py):
//
//   o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t,   S_t = diag(w_t) S_{t-1} + k_t v_t^T,   log w = -exp(z + w0)
//
//   time_mix_scan        decode rows, short spans, float32: linear_scan.cuh with the decay in the front
//   time_mix_keys        long spans: per chunk of 64 tokens the keys with their decays up to the end of the chunk, as bf16 pairs, and the
//                        chunk's decays; the states before every chunk follow from them (linear_states_per_channel)
//   time_mix_out         per chunk and head the outputs, on the tensor cores
//   tanh_rows            the decay projection's activation
//
// Inside a chunk the weight of token j's key for token i > j is, per channel, the product of the decays between them.  A chunk is cut
// into four blocks of 16 tokens.  Between blocks it factors at the block borders into parts that are at most one, r~_i = r_i times
// the decays from its block's start and k^_j = k_j times those to its block's end, with the decays of whole blocks in between.  Inside a
// block the weighted key of a column moves on from row to row, p <- p w_i, in fp32.  Nothing is divided by a decay, so strong
// ones underflow to zero and lose nothing.
#define STK_PDL_CLASS 16
#include "chunk_mma.cuh"
#include "linear_scan.cuh"
#include "pairs.cuh"

namespace stk {

template <typename A>
struct TimeMixFront {
  static constexpr bool kPerChannel = true;
  const void* proj; long long ldp; int np;        // r, k, v at columns 0, np, 2 np
  const float* z; long long ldz;
  const float* w0; const float* u;                // [H * D]
  int D;
  __device__ __forceinline__ float skip(int) const { return 0.f; }
  __device__ __forceinline__ float value(long long t, int h, int col) const {
    return ld_act(reinterpret_cast<const A*>(proj) + t * ldp + 2 * np + h * D + col);
  }
  // r and k, the bonus' u k, and the decays as a factor and what is added to it (a factor near one as 1 plus its difference from 1)
  __device__ __forceinline__ void fill(long long t, int h, float* r, float* k, float* uk, float2* w) const {
    const A* p = reinterpret_cast<const A*>(proj) + t * ldp + h * D;
    for (int d = threadIdx.x; d < D; d += kScanThreads) {
      const float kd = ld_act(p + np + d);
      r[d] = ld_act(p + d);
      k[d] = kd;
      uk[d] = u[h * D + d] * kd;
      const float g = -expf(z[t * ldz + h * D + d] + w0[h * D + d]);
      w[d] = g > -0.5f ? make_float2(1.f, expm1f(g)) : make_float2(expf(g), 0.f);
    }
  }
};

// ---- chunked form ----------------------------------------------------------------------------------
struct TmArgs {
  const __nv_bfloat16* proj; long long ldp; int np;
  const float* z; long long ldz;
  const float* w0; const float* u;
  ScanArgs s;                                     // V = D
};
constexpr int kTmSub = 16, kTmBlocks = kChunk / kTmSub;

// keys [T][2][H * D8]: high parts, remainders; channel [chunk][H][D].  One CTA per (chunk, head); a thread takes a block's 16 tokens of two
// channels.  vec: channels come in whole aligned pairs.
__global__ void __launch_bounds__(256)
time_mix_keys_kernel(const TmArgs a, int min_span, __nv_bfloat16* __restrict__ keys, int D8, float* __restrict__ channel, int vec) {
  extern __shared__ __align__(16) float ends[];   // [4][D8]
  __shared__ ChunkRef s_c;
  __shared__ int s_ok;
  pdl_wait();
  pdl_trigger();
  const int ci = blockIdx.x, h = blockIdx.y, D = a.s.D, n8 = a.s.H * D8, pairs = D8 >> 1;
  if (threadIdx.x == 0) s_ok = find_chunk(a.s.query_start, a.s.n_req, min_span, ci, s_c) ? 1 : 0;
  __syncthreads();
  if (!s_ok) return;
  const ChunkRef c = s_c;
  const int b = threadIdx.x / pairs, d = (threadIdx.x - b * pairs) * 2;      // blockDim.x = 4 * pairs
  const bool in0 = d < D, in1 = d + 1 < D;
  const float w0 = in0 ? a.w0[h * D + d] : 0.f, w1 = in1 ? a.w0[h * D + d + 1] : 0.f;
  float2 g[kTmSub], sum = make_float2(0.f, 0.f);
  __nv_bfloat162 k[kTmSub];
#pragma unroll
  for (int i = 0; i < kTmSub; ++i) {
    const int n = b * kTmSub + i;
    const long long t = c.t0 + n;
    float2 z = make_float2(0.f, 0.f);
    k[i] = __floats2bfloat162_rn(0.f, 0.f);
    if (n < c.n) {
      const float* zp = a.z + t * a.ldz + h * D + d;
      const __nv_bfloat16* kp = a.proj + t * a.ldp + a.np + h * D + d;
      if (vec && in1) {
        z = *reinterpret_cast<const float2*>(zp);
        k[i] = *reinterpret_cast<const __nv_bfloat162*>(kp);
      } else {
        if (in0) { z.x = zp[0]; k[i].x = kp[0]; }
        if (in1) { z.y = zp[1]; k[i].y = kp[1]; }
      }
    }
    g[i] = z;
  }
#pragma unroll
  for (int i = 0; i < kTmSub; ++i) {
    const bool live = b * kTmSub + i < c.n;
    g[i].x = live && in0 ? -__expf(g[i].x + w0) : 0.f;
    g[i].y = live && in1 ? -__expf(g[i].y + w1) : 0.f;
    sum.x += g[i].x;
    sum.y += g[i].y;
  }
  *reinterpret_cast<float2*>(ends + b * D8 + d) = sum;
  __syncthreads();
  float2 left = make_float2(0.f, 0.f);            // decays behind the token, up to the end of the chunk
  for (int m = kTmBlocks - 1; m > b; --m) {
    const float2 e = *reinterpret_cast<const float2*>(ends + m * D8 + d);
    left.x += e.x;
    left.y += e.y;
  }
#pragma unroll
  for (int i = kTmSub - 1; i >= 0; --i) {
    const int n = b * kTmSub + i;
    if (n < c.n) {
      const float2 kf = __bfloat1622float2(k[i]);
      uint32_t hi, lo;
      mls_split2(kf.x * __expf(left.x), kf.y * __expf(left.y), hi, lo);
      __nv_bfloat16* to = keys + (c.t0 + n) * 2 * n8 + h * D8 + d;
      *reinterpret_cast<uint32_t*>(to) = hi;
      *reinterpret_cast<uint32_t*>(to + n8) = lo;
    }
    left.x += g[i].x;
    left.y += g[i].y;
  }
  if (b == 0) {
    float* to = channel + (static_cast<long long>(ci) * a.s.H + h) * D + d;
    if (in0) to[0] = __expf(left.x);
    if (in1) to[1] = __expf(left.y);
  }
}

constexpr int kTmOutThreads = 256;
struct TmOutLayout { int ks, q, r, v, wk, w, f, p, bytes; };                      // byte offsets
__host__ __device__ inline TmOutLayout tm_out_layout(int D) {
  TmOutLayout l;
  const int Dp = blocks16(D) * 16;
  l.ks = Dp + 8;
  const int tile = kChunk * l.ks * 2, scores = 2 * kChunk * kStStride * 2;
  l.q = 0;                                        // [2][64][ks] r~ as pair
  l.r = 2 * tile;                                 // [64][ks]
  l.v = l.r + tile;                               // [64][ks]
  l.wk = l.v + tile;                              // k [64][ks], then at w decays [64][Dp] fp32; later k^ as pair [2][64][ks]; then the weighted
  l.w = l.wk + tile;                              // scores [2][64][72]
  const int first = tile + kChunk * Dp * 4, second = 2 * tile > scores ? 2 * tile : scores;
  l.f = l.wk + (first > second ? first : second); // [7][Dp] fp32: decays of blocks 1, 2, 1 and 2, 0, 0 and 1, 0 to 2; the bonus
  l.p = l.f + 7 * Dp * 4;                         // [4][Dp] sums of the blocks
  l.bytes = l.p + 4 * Dp * 4;
  return l;
}

// An operand pair times a factor per column (columns 2 (lane & 3), + 1, and 8 further).
__device__ __forceinline__ void tm_scale_pair(uint32_t (&hi)[4], uint32_t (&lo)[4], const float* f) {
  const float2 f0 = *reinterpret_cast<const float2*>(f), f1 = *reinterpret_cast<const float2*>(f + 8);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi[i]));
    const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&lo[i]));
    const float2 g = i < 2 ? f0 : f1;
    mls_split2((x.x + y.x) * g.x, (x.y + y.y) * g.y, hi[i], lo[i]);
  }
}

// One CTA per (chunk, head).
__global__ void __launch_bounds__(kTmOutThreads, 3)
time_mix_out_kernel(const TmArgs a, int min_span, const float* __restrict__ states) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ ChunkRef s_c;
  __shared__ int s_ok;
  const int D = a.s.D, nd = blocks16(D), Dp = nd * 16;
  const TmOutLayout L = tm_out_layout(D);
  const int ks = L.ks, part = kChunk * ks;
  __nv_bfloat16* q = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.q);
  __nv_bfloat16* r = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.r);
  __nv_bfloat16* v = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.v);
  __nv_bfloat16* kr = reinterpret_cast<__nv_bfloat16*>(smem_raw + L.wk);
  __nv_bfloat16* k = kr;                                                 // k^, after the keys and the decays are done with
  __nv_bfloat16* ph = kr;                                                // weighted scores, after k^
  __nv_bfloat16* pl = ph + kChunk * kStStride;
  float* w = reinterpret_cast<float*>(smem_raw + L.w);
  float* f = reinterpret_cast<float*>(smem_raw + L.f);
  float* sums = reinterpret_cast<float*>(smem_raw + L.p);
  pdl_wait();
  pdl_trigger();
  const int ci = blockIdx.x, h = blockIdx.y;
  if (threadIdx.x == 0) s_ok = find_chunk(a.s.query_start, a.s.n_req, min_span, ci, s_c) ? 1 : 0;
  __syncthreads();
  if (!s_ok) return;
  const ChunkRef c = s_c;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const __nv_bfloat16* p = a.proj + c.t0 * a.ldp + h * D;
  load_rows_async(r, ks, Dp, p, a.ldp, c.n, D, kTmOutThreads);
  load_rows_async(kr, ks, Dp, p + a.np, a.ldp, c.n, D, kTmOutThreads);
  load_rows_async(v, ks, Dp, p + 2 * a.np, a.ldp, c.n, D, kTmOutThreads);
  mls_commit();
  for (int d = threadIdx.x; d < Dp; d += kTmOutThreads) f[6 * Dp + d] = d < D ? a.u[h * D + d] : 0.f;
  // a thread's (block, channel) in every round: at most two rounds, up to 128 channels
  float g[2][kTmSub];
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    const int e = threadIdx.x + m * kTmOutThreads, b = e / Dp, d = e - b * Dp;
    const bool in = e < kTmBlocks * Dp && d < D;
    if (m > 0 && Dp <= 64) continue;
    const float w0 = in ? a.w0[h * D + d] : 0.f;
#pragma unroll
    for (int i = 0; i < kTmSub; ++i) g[m][i] = in && b * kTmSub + i < c.n ? a.z[(c.t0 + b * kTmSub + i) * a.ldz + h * D + d] : 0.f;
#pragma unroll
    for (int i = 0; i < kTmSub; ++i) g[m][i] = in && b * kTmSub + i < c.n ? -__expf(g[m][i] + w0) : 0.f;
    if (e < kTmBlocks * Dp) {
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < kTmSub; ++i) {
        w[(b * kTmSub + i) * Dp + d] = __expf(g[m][i]);
        sum += g[m][i];
      }
      sums[b * Dp + d] = sum;
    }
  }
  mls_wait<0>();
  __syncthreads();
  for (int d = threadIdx.x; d < Dp; d += kTmOutThreads) {
    const float s0 = sums[d], s1 = sums[Dp + d], s2 = sums[2 * Dp + d];
    f[d] = __expf(s1);
    f[Dp + d] = __expf(s2);
    f[2 * Dp + d] = __expf(s1 + s2);
    f[3 * Dp + d] = __expf(s0);
    f[4 * Dp + d] = __expf(s0 + s1);
    f[5 * Dp + d] = __expf(s0 + s1 + s2);
  }
  // the blocks on the diagonal: four lanes per column, each four channels of every 16
  float acc[kTmSub], bonus = 0.f;
  const int jb = warp >> 1, j = (warp & 1) * 8 + (lane >> 2), seg = lane & 3;
#pragma unroll
  for (int i = 0; i < kTmSub; ++i) acc[i] = 0.f;
  for (int c0 = seg * 4; c0 < Dp; c0 += 16) {
    const uint2 kv = *reinterpret_cast<const uint2*>(kr + (jb * kTmSub + j) * ks + c0);
    const uint2 rv = *reinterpret_cast<const uint2*>(r + (jb * kTmSub + j) * ks + c0);
    uint64_t x0 = widen2(kv.x), x1 = widen2(kv.y);
    const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(f + 6 * Dp + c0);
    float s0, s1;
    unpack2(fma2(mul2(widen2(rv.x), u.x), x0, mul2(mul2(widen2(rv.y), u.y), x1)), s0, s1);
    bonus += s0 + s1;
#pragma unroll
    for (int i = 1; i < kTmSub; ++i) {
      if (i < 9 && (warp & 1)) continue;                                 // the warp's columns start behind these rows
      const ulonglong2 wi = *reinterpret_cast<const ulonglong2*>(w + (jb * kTmSub + i) * Dp + c0);
      const uint2 y = *reinterpret_cast<const uint2*>(r + (jb * kTmSub + i) * ks + c0);
      unpack2(fma2(widen2(y.x), x0, mul2(widen2(y.y), x1)), s0, s1);
      const bool below = i > j;
      acc[i] += below ? s0 + s1 : 0.f;
      x0 = below ? mul2(x0, wi.x) : x0;
      x1 = below ? mul2(x1, wi.y) : x1;
    }
  }
  bonus += __shfl_xor_sync(0xffffffffu, bonus, 1);
  bonus += __shfl_xor_sync(0xffffffffu, bonus, 2);
  // k^ of every block in registers, r~ to its place
  uint32_t kh[2][kTmSub / 2], kl[2][kTmSub / 2];                         // two tokens each
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    const int e = threadIdx.x + m * kTmOutThreads, b = e / Dp, d = e - b * Dp;
    if ((m > 0 && Dp <= 64) || e >= kTmBlocks * Dp) continue;
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < kTmSub; ++i) {
      const int n = b * kTmSub + i;
      mls_split(bf16_to_f(r[n * ks + d]) * __expf(sum), q[n * ks + d], q[part + n * ks + d]);
      sum += g[m][i];
    }
    float left = 0.f;
#pragma unroll
    for (int i = kTmSub / 2 - 1; i >= 0; --i) {
      const int n = b * kTmSub + 2 * i;
      const float y1 = bf16_to_f(kr[(n + 1) * ks + d]) * __expf(left);
      left += g[m][2 * i + 1];
      const float y0 = bf16_to_f(kr[n * ks + d]) * __expf(left);
      left += g[m][2 * i];
      mls_split2(y0, y1, kh[m][i], kl[m][i]);
    }
  }
#pragma unroll
  for (int i = 0; i < kTmSub; ++i) {
    acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], 1);
    acc[i] += __shfl_xor_sync(0xffffffffu, acc[i], 2);
  }
  __syncthreads();                                                       // keys and decays are done with
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    const int e = threadIdx.x + m * kTmOutThreads, b = e / Dp, d = e - b * Dp;
    if ((m > 0 && Dp <= 64) || e >= kTmBlocks * Dp) continue;
#pragma unroll
    for (int i = 0; i < kTmSub / 2; ++i) {
      __nv_bfloat16* to = k + (b * kTmSub + 2 * i) * ks + d;
      const __nv_bfloat162 hi = *reinterpret_cast<const __nv_bfloat162*>(&kh[m][i]), lo = *reinterpret_cast<const __nv_bfloat162*>(&kl[m][i]);
      to[0] = hi.x;
      to[ks] = hi.y;
      to[part] = lo.x;
      to[part + ks] = lo.y;
    }
  }
  __syncthreads();
  // the six blocks below the diagonal, one per warp
  uint32_t wh[4], wl[4];
  int rb = 0, kb = 0;
  if (warp < 6) {
    rb = warp < 1 ? 1 : warp < 3 ? 2 : 3;
    kb = warp - rb * (rb - 1) / 2;
    const float* g = rb - kb == 1 ? nullptr : rb - kb == 3 ? f + 2 * Dp : kb == 0 ? f : f + Dp;
    float x[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) x[n][i] = 0.f;
    const int qo = (rb * 16 + (lane & 15)) * ks + (lane >> 4) * 8;
    const int ko = (kb * 16 + (lane >> 4) * 8 + (lane & 7)) * ks + ((lane >> 3) & 1) * 8;
    for (int kk = 0; kk < nd; ++kk) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      mls_ldsm4(ah, q + qo + kk * 16);
      mls_ldsm4(al, q + part + qo + kk * 16);
      mls_ldsm4(bh, k + ko + kk * 16);
      mls_ldsm4(bl, k + part + ko + kk * 16);
      if (g != nullptr) tm_scale_pair(ah, al, g + kk * 16 + (lane & 3) * 2);
      mls_mma(x[0], ah, bh[0], bh[1]);
      mls_mma(x[1], ah, bh[2], bh[3]);
      mls_mma(x[0], al, bh[0], bh[1]);
      mls_mma(x[1], al, bh[2], bh[3]);
      mls_mma(x[0], ah, bl[0], bl[1]);
      mls_mma(x[1], ah, bl[2], bl[3]);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 2; ++i) mls_split2(x[n][2 * i], x[n][2 * i + 1], wh[2 * n + i], wl[2 * n + i]);
  }
  __syncthreads();                                                       // k^ is done with
  if (warp < 6) {
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int off = (rb * 16 + (lane >> 2) + i * 8) * kStStride + kb * 16 + n * 8 + (lane & 3) * 2;
        *reinterpret_cast<uint32_t*>(ph + off) = wh[2 * n + i];
        *reinterpret_cast<uint32_t*>(pl + off) = wl[2 * n + i];
      }
  }
#pragma unroll
  for (int i = 0; i < kTmSub; ++i) {
    if ((i & 3) != seg) continue;
    const int off = (jb * kTmSub + i) * kStStride + jb * kTmSub + j;
    mls_split(i > j ? acc[i] : i == j ? bonus : 0.f, ph[off], pl[off]);
  }
  const bool has_state = !(a.s.start_pos[c.ri] == 0 && c.first == ci);
  if (has_state) {
    // r~ decayed from the chunk's start on, for the state: blocks 1 to 3
    const int per = Dp / 8;
    for (int e = threadIdx.x; e < 48 * per; e += kTmOutThreads) {
      const int t = e / per + 16, c0 = (e % per) * 8;
      uint4* at = reinterpret_cast<uint4*>(q + t * ks + c0);
      uint4* rest = reinterpret_cast<uint4*>(q + part + t * ks + c0);
      const ulonglong2* by = reinterpret_cast<const ulonglong2*>(f + (2 + (t >> 4)) * Dp + c0);
      const ulonglong2 g0 = by[0], g1 = by[1];
      uint4 hi = *at, lo = *rest;
      auto scale = [&](uint32_t& x, uint32_t& y, uint64_t g) {
        float s0, s1;
        unpack2(mul2(add2(widen2(x), widen2(y)), g), s0, s1);
        mls_split2(s0, s1, x, y);
      };
      scale(hi.x, lo.x, g0.x);
      scale(hi.y, lo.y, g0.y);
      scale(hi.z, lo.z, g1.x);
      scale(hi.w, lo.w, g1.y);
      *at = hi;
      *rest = lo;
    }
  }
  __syncthreads();                                                       // the weighted scores are complete
  const uint4* S0 = reinterpret_cast<const uint4*>(states + (static_cast<long long>(ci) * a.s.H + h) * linear_slot_floats(D, D)) + lane;
  for (int unit = warp; unit < 2 * nd; unit += kTmOutThreads / 32) {     // 16 columns, 32 rows
    const int cg = unit >> 1, rh = unit & 1;
    float o[2][2][4];
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int y = 0; y < 2; ++y)
#pragma unroll
        for (int i = 0; i < 4; ++i) o[x][y][i] = 0.f;
    if (has_state) {
      const uint4* S = S0 + static_cast<long long>(cg) * nd * 64;
#pragma unroll 4
      for (int kk = 0; kk < nd; ++kk) {
        const uint4 hi = __ldcs(S + kk * 64), lo = __ldcs(S + kk * 64 + 32);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int rb2 = rh * 2 + x;
          uint32_t ah[4], al[4];
          const int qo = (rb2 * 16 + (lane & 15)) * ks + (lane >> 4) * 8 + kk * 16;
          mls_ldsm4(ah, q + qo);
          mls_ldsm4(al, q + part + qo);
          mls_mma(o[x][0], ah, hi.x, hi.y);
          mls_mma(o[x][1], ah, hi.z, hi.w);
          mls_mma(o[x][0], ah, lo.x, lo.y);
          mls_mma(o[x][1], ah, lo.z, lo.w);
          mls_mma(o[x][0], al, hi.x, hi.y);
          mls_mma(o[x][1], al, hi.z, hi.w);
        }
      }
    }
    for (int b = 0; b <= rh * 2 + 1; ++b) {
      uint32_t bv[4];
      mls_ldsm4_t(bv, v + (b * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ks + cg * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int rb2 = rh * 2 + x;
        if (b > rb2) continue;
        uint32_t hi[4], lo[4];
        const int off = (rb2 * 16 + (lane & 15)) * kStStride + b * 16 + (lane >> 4) * 8;
        mls_ldsm4(hi, ph + off);
        mls_ldsm4(lo, pl + off);
        mls_mma(o[x][0], hi, bv[0], bv[1]);
        mls_mma(o[x][1], hi, bv[2], bv[3]);
        mls_mma(o[x][0], lo, bv[0], bv[1]);
        mls_mma(o[x][1], lo, bv[2], bv[3]);
      }
    }
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = (rh * 2 + x) * 16 + (lane >> 2) + i * 8;
        if (t >= c.n) continue;
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          const int col = cg * 16 + y * 8 + (lane & 3) * 2;
          float* to = a.s.o + ((c.t0 + t) * static_cast<long long>(a.s.H) + h) * D + col;
          if ((D & 1) == 0 && col + 1 < D) {
            *reinterpret_cast<float2*>(to) = make_float2(o[x][y][2 * i], o[x][y][2 * i + 1]);
          } else {
            if (col < D) to[0] = o[x][y][2 * i];
            if (col + 1 < D) to[1] = o[x][y][2 * i + 1];
          }
        }
      }
  }
}

// tanh of fp32 rows; kPair: bf16 high parts, then the remainders n columns further.
template <bool kPair>
__global__ void __launch_bounds__(256)
tanh_rows_kernel(const float* __restrict__ z, long long ldz, int n, void* __restrict__ out, long long total) {
  pdl_wait();
  pdl_trigger();
  const long long e = blockIdx.x * 256ll + threadIdx.x;
  if (e >= total) return;
  const long long t = e / n;
  const int c = static_cast<int>(e - t * n);
  const float y = tanhf(z[t * ldz + c]);
  if (kPair) {
    __nv_bfloat16* o = reinterpret_cast<__nv_bfloat16*>(out) + t * 2 * n + c;
    const __nv_bfloat16 hi = __float2bfloat16(y);
    o[0] = hi;
    o[n] = __float2bfloat16(y - bf16_to_f(hi));
  } else {
    reinterpret_cast<float*>(out)[t * n + c] = y;
  }
}

}  // namespace stk

using namespace stk;

// Spans of min_span .. max_span tokens, token by token.
STK_API int stk_time_mix_scan(const void* proj, long long ldp, int np, const float* z, long long ldz, const float* w0, const float* u,
                              const int* query_start, const int* req_rows, const int* start_pos, int n_req, float* S, float* o, int heads,
                              int dim, int fp32, int min_span, int max_span, int T, void* stream) {
  if (T <= 0) return 0;
  const ScanArgs a{query_start, req_rows, start_pos, n_req, S, o, heads, dim, dim};
  if (fp32) return launch_scan(TimeMixFront<float>{proj, ldp, np, z, ldz, w0, u, dim}, a, min_span, max_span, (cudaStream_t)stream);
  return launch_scan(TimeMixFront<__nv_bfloat16>{proj, ldp, np, z, ldz, w0, u, dim}, a, min_span, max_span, (cudaStream_t)stream);
}

// out [T, n] fp32, or [T, 2 n] bf16: high parts and remainders.
STK_API int stk_tanh_rows(const float* z, long long ldz, int n, void* out, int fp32, int T, void* stream) {
  if (T <= 0 || n <= 0) return 0;
  const long long total = static_cast<long long>(T) * n;
  const dim3 grid(static_cast<unsigned>((total + 255) / 256));
  if (fp32) launch_pdl(tanh_rows_kernel<false>, grid, dim3(256), 0, (cudaStream_t)stream, z, ldz, n, out, total);
  else launch_pdl(tanh_rows_kernel<true>, grid, dim3(256), 0, (cudaStream_t)stream, z, ldz, n, out, total);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// Whether `stk_time_mix_chunks` covers a head size.
STK_API int stk_time_mix_chunks_ok(int dim) { return dim >= 1 && dim <= 128 ? 1 : 0; }

// Spans of at least min_span tokens, bf16.  keys: work space [T, 2, heads * d8] bf16 (d8: dim rounded up to 8); channel: fp32
// [max_chunks, heads, dim]; states: fp32 [max_chunks * heads * stk_linear_state_slot()]; max_chunks bounds the chunks over all requests.
STK_API int stk_time_mix_chunks(const void* proj, long long ldp, int np, const float* z, long long ldz, const float* w0, const float* u,
                                const int* query_start, const int* req_rows, const int* start_pos, int n_req, float* S, float* o, int heads,
                                int dim, int min_span, void* keys, float* channel, float* states, int max_chunks, int T, void* stream) {
  if (T <= 0 || n_req <= 0 || max_chunks <= 0) return 0;
  if (!stk_time_mix_chunks_ok(dim) || heads < 1 || static_cast<long long>(heads) * n_req > 65535 || min_span < 1 ||
      ((reinterpret_cast<uintptr_t>(states) | reinterpret_cast<uintptr_t>(keys)) & 15))
    return -1;
  const int d8 = (dim + 7) / 8 * 8, n8 = heads * d8;
  const int vec = dim % 2 == 0 && ldp % 2 == 0 && np % 2 == 0 && ldz % 2 == 0 && (reinterpret_cast<uintptr_t>(proj) & 3) == 0 &&
                  (reinterpret_cast<uintptr_t>(z) & 7) == 0;
  TmArgs a;
  a.proj = (const __nv_bfloat16*)proj; a.ldp = ldp; a.np = np; a.z = z; a.ldz = ldz; a.w0 = w0; a.u = u;
  a.s = ScanArgs{query_start, req_rows, start_pos, n_req, S, o, heads, dim, dim};
  cudaStream_t st = (cudaStream_t)stream;
  __nv_bfloat16* kp = (__nv_bfloat16*)keys;
  launch_pdl(time_mix_keys_kernel, dim3(max_chunks, heads), dim3(2 * d8), static_cast<size_t>(kTmBlocks) * d8 * sizeof(float), st, a, min_span, kp,
             d8, channel, vec);
  const int rc = linear_states_per_channel(kp, kp + n8, 2ll * n8, d8, d8, a.proj, ldp, 2 * np, channel, a.s, min_span, states, T, st);
  if (rc != 0) return rc;
  if (cudaFuncSetAttribute(time_mix_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return -3;
  launch_pdl(time_mix_out_kernel, dim3(max_chunks, heads), dim3(kTmOutThreads), static_cast<size_t>(tm_out_layout(dim).bytes), st, a, min_span,
             (const float*)states);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
