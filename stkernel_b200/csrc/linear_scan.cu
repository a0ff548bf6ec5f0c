// Chunked form of the linear recurrences with a scalar decay (linear_scan.cuh) for bf16 operands: with F the running sum of g inside
// a chunk of 64 tokens and w the tokens' input weights,
//
//   o_t   = exp(F_t) S_start^T q_t + sum_{j <= t} exp(F_t - F_j) w_j (k_j . q_t) v_j  (+ skip v_t)
//   S_end = exp(F_end) S_start + sum_j exp(F_end - F_j) w_j k_j v_j^T
//
//   linear_chunk_state     one CTA per 64 x 64 block of a head's state walks the chunks of a request with the block in its
//                          accumulators and leaves the state before each chunk as bf16 pairs (high part and remainder)
//   linear_chunk_out       per chunk, head and 64 or 128 value columns: the outputs
//
// Both run on the tensor cores.  fp32 operands (weighted keys, weighted scores, the state; queries and keys where they come as
// pairs) enter the products as bf16 pairs, so they keep 16 mantissa bits.
#define STK_PDL_CLASS 16
#include "chunk_mma.cuh"
#include "linear_scan.cuh"

namespace stk {

typedef __nv_bfloat16 bf16;

struct ChunkArgs {
  const bf16* qh; const bf16* ql; const bf16* kh; const bf16* kl;     // remainders may be null
  long long ldqk; int step, width, hpg;          // row stride, columns per head (group of hpg heads), columns used of them
  const bf16* v; long long ldv; int v_off;
  const float* fixed;                            // [H] log decay of every token, or
  const float* g; const float* w;                // [H, T] log decay and input weight
  const float* skip;                             // [H] or null
  ScanArgs s;
  int T;
};

// A chunk's state before its first token: [D][Vp] high parts, then [D][Vp] remainders; Vp = V rounded up to 8.
__host__ __device__ inline long long linear_slot_floats(int D, int V) {
  return (static_cast<long long>(D) * ((V + 7) / 8 * 8) + 3) / 4 * 4;
}

// Tokens 2 * lane and 2 * lane + 1 of a chunk of n: running sums of the log decays (F) and input weights (w, 0 behind the chunk).
struct ChunkGates { float F0, F1, w0, w1, end; };
struct ChunkRaw { float g0, g1, w0, w1; };

__device__ __forceinline__ ChunkRaw load_gates(const ChunkArgs& a, int h, long long t0, int n, int lane) {
  ChunkRaw r = {0.f, 0.f, 1.f, 1.f};
  if (a.fixed != nullptr) {
    r.g0 = r.g1 = a.fixed[h];
  } else {
    const long long at = static_cast<long long>(h) * a.T + t0 + 2 * lane;
    if (2 * lane < n) { r.g0 = a.g[at]; r.w0 = a.w[at]; }
    if (2 * lane + 1 < n) { r.g1 = a.g[at + 1]; r.w1 = a.w[at + 1]; }
  }
  return r;
}
__device__ __forceinline__ ChunkGates chunk_gates(const ChunkArgs& a, const ChunkRaw& r, int n, int lane) {
  ChunkGates c;
  if (a.fixed != nullptr) {
    c.F0 = r.g0 * static_cast<float>(2 * lane + 1);
    c.F1 = r.g0 * static_cast<float>(2 * lane + 2);
    c.end = r.g0 * static_cast<float>(n);
  } else {
    const float pair = r.g0 + r.g1;
    float inc = pair;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += up;
    }
    c.F0 = inc - r.g1;
    c.F1 = inc;
    c.end = __shfl_sync(0xffffffffu, inc, 31);                          // absent tokens add nothing
  }
  c.w0 = 2 * lane < n ? r.w0 : 0.f;
  c.w1 = 2 * lane + 1 < n ? r.w1 : 0.f;
  return c;
}

template <bool kPair>
__global__ void __launch_bounds__(128)
linear_chunk_state_kernel(const ChunkArgs a, int min_span, float* __restrict__ states) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ float s_w[kChunk];
  __shared__ float s_fs;
  constexpr int kTile = kChunk * kStStride, kParts = kPair ? 2 : 1;
  bf16* kt = reinterpret_cast<bf16*>(smem_raw);                         // [2 stages][parts][64 tokens][72]
  bf16* vt = kt + 2 * kParts * kTile;                                   // [2 stages][64][72]
  bf16* wh = vt + 2 * kTile;                                            // weighted keys, high part
  bf16* wl = wh + kTile;                                                // remainder
  pdl_wait();
  pdl_trigger();
  const ScanArgs& s = a.s;
  const int vb = blockIdx.x, db = blockIdx.y, h = blockIdx.z % s.H, ri = blockIdx.z / s.H;
  const int q0 = s.query_start[ri], span = s.query_start[ri + 1] - q0;
  if (span < min_span || span <= 0) return;
  const int first = first_chunk(s.query_start, min_span, ri), nc = (span + kChunk - 1) / kChunk;
  const long long row = s.req_rows[ri];
  const bool fresh = s.start_pos[ri] == 0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int d0 = db * 64 + warp * 16 + (lane >> 2), c0 = vb * 64 + (lane & 3) * 2;
  const int Vp = (s.V + 7) / 8 * 8;
  const long long slot_f = linear_slot_floats(s.D, s.V);
  float* gS = s.S + (row * s.H + h) * static_cast<long long>(s.D) * s.V;
  const int kn = max(0, min(64, a.width - db * 64)), vn = min(64, s.V - vb * 64);
  float acc[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = d0 + (i >> 1) * 8, c = c0 + j * 8 + (i & 1);
      acc[j][i] = !fresh && d < s.D && c < s.V ? gS[static_cast<long long>(d) * s.V + c] : 0.f;
    }
  const int kc = h / a.hpg * a.step + db * 64;
  auto load = [&](int c) {
    const int n = min(kChunk, span - c * kChunk), st = c & 1;
    const long long t0 = q0 + c * kChunk;
    load_rows_async(kt + st * kParts * kTile, kStStride, 64, a.kh + t0 * a.ldqk + kc, a.ldqk, n, kn, 128);
    if (kPair) load_rows_async(kt + (st * kParts + 1) * kTile, kStStride, 64, a.kl + t0 * a.ldqk + kc, a.ldqk, n, kn, 128);
    load_rows_async(vt + st * kTile, kStStride, 64, a.v + t0 * a.ldv + a.v_off + h * s.V + vb * 64, a.ldv, n, vn, 128);
  };
  ChunkRaw raw = {};
  load(0);
  mls_commit();
  if (warp == 0) raw = load_gates(a, h, q0, min(kChunk, span), lane);
  for (int c = 0; c < nc; ++c) {
    const int n = min(kChunk, span - c * kChunk);
    if (warp == 0) {
      const ChunkGates g = chunk_gates(a, raw, n, lane);
      s_w[2 * lane] = 2 * lane < n ? g.w0 * expf(g.end - g.F0) : 0.f;
      s_w[2 * lane + 1] = 2 * lane + 1 < n ? g.w1 * expf(g.end - g.F1) : 0.f;
      if (lane == 0) s_fs = expf(g.end);
    }
    if (c + 1 < nc) load(c + 1);
    mls_commit();
    mls_wait<1>();
    __syncthreads();
    if (warp == 0 && c + 1 < nc) raw = load_gates(a, h, q0 + (c + 1) * kChunk, min(kChunk, span - (c + 1) * kChunk), lane);
    // the state before this chunk
    {
      bf16* sh = reinterpret_cast<bf16*>(states + (static_cast<long long>(first + c) * s.H + h) * slot_f);
      bf16* sl = sh + static_cast<long long>(s.D) * Vp;
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int d = d0 + r * 8, col = c0 + j * 8;
          if (d < s.D && col < Vp) {
            uint32_t hi, lo;
            mls_split2(acc[j][2 * r], acc[j][2 * r + 1], hi, lo);
            *reinterpret_cast<uint32_t*>(sh + static_cast<long long>(d) * Vp + col) = hi;
            *reinterpret_cast<uint32_t*>(sl + static_cast<long long>(d) * Vp + col) = lo;
          }
        }
    }
    const bf16* k = kt + (c & 1) * kParts * kTile;
    const bf16* v = vt + (c & 1) * kTile;
    for (int e = threadIdx.x; e < kChunk * 32; e += 128) {
      const int r = e >> 5, cc = (e & 31) * 2;
      float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k + r * kStStride + cc));
      if (kPair) {
        const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(k + kTile + r * kStStride + cc));
        x.x += y.x;
        x.y += y.y;
      }
      const float w = s_w[r];
      uint32_t hi, lo;
      mls_split2(x.x * w, x.y * w, hi, lo);
      *reinterpret_cast<uint32_t*>(wh + r * kStStride + cc) = hi;
      *reinterpret_cast<uint32_t*>(wl + r * kStStride + cc) = lo;
    }
    const float fs = s_fs;
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[j][i] *= fs;
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kChunk / 16; ++kk) {
      uint32_t ah[4], al[4];
      const int ao = (kk * 16 + (lane & 7) + (lane >> 4) * 8) * kStStride + warp * 16 + ((lane >> 3) & 1) * 8;
      mls_ldsm4_t(ah, wh + ao);
      mls_ldsm4_t(al, wl + ao);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        uint32_t b[4];
        mls_ldsm4_t(b, v + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kStStride + j * 16 + (lane >> 4) * 8);
        mls_mma(acc[2 * j], ah, b[0], b[1]);
        mls_mma(acc[2 * j + 1], ah, b[2], b[3]);
        mls_mma(acc[2 * j], al, b[0], b[1]);
        mls_mma(acc[2 * j + 1], al, b[2], b[3]);
      }
    }
    __syncthreads();
  }
  mls_wait<0>();
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = d0 + (i >> 1) * 8, c = c0 + j * 8 + (i & 1);
      if (d < s.D && c < s.V) gS[static_cast<long long>(d) * s.V + c] = acc[j][i];
    }
}

constexpr int kLoRows = 32;                      // state rows per stage

// Eight warps: four blocks of 16 tokens x two halves of the columns (of the keys while the scores are formed).
template <bool kPair, int COLS>
__global__ void __launch_bounds__(256)
linear_chunk_out_kernel(const ChunkArgs a, int min_span, const float* __restrict__ states) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ float s_F[kChunk], s_w[kChunk], s_in[kChunk];
  __shared__ ChunkRef s_c;
  __shared__ int s_ok;
  constexpr int kVs = COLS + 8, kHalf = COLS / 2, kParts = kPair ? 2 : 1;
  const ScanArgs& s = a.s;
  const int Dp = (s.D + 15) / 16 * 16, ks = Dp + 8;
  bf16* q = reinterpret_cast<bf16*>(smem_raw);                          // [parts][64][Dp + 8]
  bf16* v = q + kParts * kChunk * ks;                                   // [64][COLS + 8]
  bf16* ph = v + kChunk * kVs;                                          // [64][72] weighted scores, high part
  bf16* pl = ph + kChunk * kStStride;                                   // remainder
  bf16* k = pl + kChunk * kStStride;                                    // [parts][64][Dp + 8], then two stages of state rows:
  bf16* st = k;                                                         // {high, remainder} x [32][COLS + 8]
  pdl_wait();
  pdl_trigger();
  const int vb = blockIdx.x, ci = blockIdx.y, h = blockIdx.z;
  if (threadIdx.x == 0) s_ok = find_chunk(s.query_start, s.n_req, min_span, ci, s_c) ? 1 : 0;
  __syncthreads();
  if (!s_ok) return;
  const ChunkRef c = s_c;
  const int Vp = (s.V + 7) / 8 * 8, qc = h / a.hpg * a.step, vn = min(COLS, s.V - vb * COLS);
  const bf16* Sh = reinterpret_cast<const bf16*>(states + (static_cast<long long>(ci) * s.H + h) * linear_slot_floats(s.D, s.V));
  const bf16* Sl = Sh + static_cast<long long>(s.D) * Vp;
  // a request's very first chunk starts from zeros: nothing comes from the state
  const bool has_state = !(s.start_pos[c.ri] == 0 && c.first == ci);
  const long long at = c.t0 * a.ldqk + qc;
  load_rows_async(q, ks, Dp, a.qh + at, a.ldqk, c.n, a.width, 256);
  load_rows_async(k, ks, Dp, a.kh + at, a.ldqk, c.n, a.width, 256);
  if (kPair) {
    load_rows_async(q + kChunk * ks, ks, Dp, a.ql + at, a.ldqk, c.n, a.width, 256);
    load_rows_async(k + kChunk * ks, ks, Dp, a.kl + at, a.ldqk, c.n, a.width, 256);
  }
  load_rows_async(v, kVs, COLS, a.v + c.t0 * a.ldv + a.v_off + h * s.V + vb * COLS, a.ldv, c.n, vn, 256);
  mls_commit();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rb = warp & 3, half = warp >> 2;
  if (warp == 0) {
    const ChunkGates g = chunk_gates(a, load_gates(a, h, c.t0, c.n, lane), c.n, lane);
    s_F[2 * lane] = g.F0;
    s_F[2 * lane + 1] = g.F1;
    s_w[2 * lane] = g.w0;
    s_w[2 * lane + 1] = g.w1;
    s_in[2 * lane] = expf(g.F0);
    s_in[2 * lane + 1] = expf(g.F1);
  }
  mls_wait<0>();
  __syncthreads();
  int row[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) row[r] = rb * 16 + (lane >> 2) + r * 8;
  // weighted scores of this warp's tokens against every other block of 16 keys
  {
    const float F[2] = {s_F[row[0]], s_F[row[1]]};
    for (int kb = half; kb <= rb; kb += 2) {
      float x[2][4];
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) x[j][i] = 0.f;
      const int qo = (rb * 16 + (lane & 15)) * ks + (lane >> 4) * 8;
      const int ko = (kb * 16 + (lane >> 4) * 8 + (lane & 7)) * ks + ((lane >> 3) & 1) * 8;
      for (int kk = 0; kk < Dp / 16; ++kk) {
        uint32_t af[4], bf[4];
        mls_ldsm4(af, q + qo + kk * 16);
        mls_ldsm4(bf, k + ko + kk * 16);
        mls_mma(x[0], af, bf[0], bf[1]);
        mls_mma(x[1], af, bf[2], bf[3]);
        if (kPair) {
          uint32_t al[4], bl[4];
          mls_ldsm4(al, q + kChunk * ks + qo + kk * 16);
          mls_ldsm4(bl, k + kChunk * ks + ko + kk * 16);
          mls_mma(x[0], al, bf[0], bf[1]);
          mls_mma(x[1], al, bf[2], bf[3]);
          mls_mma(x[0], af, bl[0], bl[1]);
          mls_mma(x[1], af, bl[2], bl[3]);
        }
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int col = kb * 16 + j * 8 + (lane & 3) * 2;
          float p[2];
#pragma unroll
          for (int i = 0; i < 2; ++i)
            p[i] = col + i <= row[r] ? x[j][2 * r + i] * (s_w[col + i] * expf(F[r] - s_F[col + i])) : 0.f;
          uint32_t hi, lo;
          mls_split2(p[0], p[1], hi, lo);
          *reinterpret_cast<uint32_t*>(ph + row[r] * kStStride + col) = hi;
          *reinterpret_cast<uint32_t*>(pl + row[r] * kStStride + col) = lo;
        }
    }
  }
  __syncthreads();                                                       // k is free, the weighted scores are complete
  float o[COLS / 16][4];
#pragma unroll
  for (int j = 0; j < COLS / 16; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[j][i] = 0.f;
  if (has_state) {
    const int slices = (Dp + kLoRows - 1) / kLoRows;
    constexpr int kCh = COLS / 8;
    auto load_slice = [&](int sl) {
      bf16* dst = st + (sl & 1) * 2 * kLoRows * kVs;
      for (int e = threadIdx.x; e < 2 * kLoRows * kCh; e += 256) {
        const int part = e / (kLoRows * kCh), r = e / kCh % kLoRows, cc = e % kCh * 8;
        const int d = sl * kLoRows + r, col = vb * COLS + cc;
        const bool ok = d < s.D && col < Vp;
        const bf16* src = (part ? Sl : Sh) + (ok ? static_cast<long long>(d) * Vp + col : 0);
        mls_cp16(dst + (part * kLoRows + r) * kVs + cc, src, ok);
      }
    };
    load_slice(0);
    mls_commit();
    for (int sl = 0; sl < slices; ++sl) {
      if (sl + 1 < slices) load_slice(sl + 1);
      mls_commit();
      mls_wait<1>();
      __syncthreads();
      const bf16* hi = st + (sl & 1) * 2 * kLoRows * kVs;
      const bf16* lo = hi + kLoRows * kVs;
#pragma unroll
      for (int kk = 0; kk < kLoRows / 16; ++kk) {
        if (sl * kLoRows + kk * 16 < Dp) {
          uint32_t af[4], al[4];
          const int qo = (rb * 16 + (lane & 15)) * ks + sl * kLoRows + kk * 16 + (lane >> 4) * 8;
          mls_ldsm4(af, q + qo);
          if (kPair) mls_ldsm4(al, q + kChunk * ks + qo);
#pragma unroll
          for (int j = 0; j < COLS / 32; ++j) {
            uint32_t bh[4], bl[4];
            const int off = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kVs + half * kHalf + j * 16 + (lane >> 4) * 8;
            mls_ldsm4_t(bh, hi + off);
            mls_ldsm4_t(bl, lo + off);
            mls_mma(o[2 * j], af, bh[0], bh[1]);
            mls_mma(o[2 * j + 1], af, bh[2], bh[3]);
            mls_mma(o[2 * j], af, bl[0], bl[1]);
            mls_mma(o[2 * j + 1], af, bl[2], bl[3]);
            if (kPair) {
              mls_mma(o[2 * j], al, bh[0], bh[1]);
              mls_mma(o[2 * j + 1], al, bh[2], bh[3]);
            }
          }
        }
      }
      __syncthreads();
    }
    mls_wait<0>();
#pragma unroll
    for (int j = 0; j < COLS / 16; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) o[j][i] *= s_in[row[i >> 1]];
  }
  for (int kb = 0; kb <= rb; ++kb) {
    uint32_t hi[4], lo[4];
    const int off = (rb * 16 + (lane & 15)) * kStStride + kb * 16 + (lane >> 4) * 8;
    mls_ldsm4(hi, ph + off);
    mls_ldsm4(lo, pl + off);
#pragma unroll
    for (int j = 0; j < COLS / 32; ++j) {
      uint32_t bf[4];
      mls_ldsm4_t(bf, v + (kb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kVs + half * kHalf + j * 16 + (lane >> 4) * 8);
      mls_mma(o[2 * j], hi, bf[0], bf[1]);
      mls_mma(o[2 * j + 1], hi, bf[2], bf[3]);
      mls_mma(o[2 * j], lo, bf[0], bf[1]);
      mls_mma(o[2 * j + 1], lo, bf[2], bf[3]);
    }
  }
  const float skip = a.skip != nullptr ? a.skip[h] : 0.f;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    if (row[r] >= c.n) continue;
    const long long t = c.t0 + row[r];
    const int lc = half * kHalf + (lane & 3) * 2, c0 = vb * COLS + lc;
    float* out = s.o + (t * s.H + h) * s.V + c0;
    const bool pair = (s.V & 1) == 0;
#pragma unroll
    for (int j = 0; j < COLS / 16; ++j) {
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v + row[r] * kVs + lc + j * 8));
      const float y0 = fmaf(skip, x.x, o[j][2 * r]), y1 = fmaf(skip, x.y, o[j][2 * r + 1]);
      if (pair && c0 + j * 8 + 1 < s.V) {
        *reinterpret_cast<float2*>(out + j * 8) = make_float2(y0, y1);
      } else {
        if (c0 + j * 8 < s.V) out[j * 8] = y0;
        if (c0 + j * 8 + 1 < s.V) out[j * 8 + 1] = y1;
      }
    }
  }
}

template <bool kPair, int COLS>
static int launch_chunks(const ChunkArgs& a, int min_span, float* states, int max_chunks, cudaStream_t st) {
  constexpr int kParts = kPair ? 2 : 1, kVs = COLS + 8;
  const ScanArgs& s = a.s;
  const int ks = (s.D + 15) / 16 * 16 + 8;
  const size_t smem_s = static_cast<size_t>(2 * kParts + 2 + 2) * kChunk * kStStride * 2;
  const size_t keys = static_cast<size_t>(kParts) * kChunk * ks, rows = static_cast<size_t>(4) * kLoRows * kVs;
  const size_t smem_o = (keys + static_cast<size_t>(kChunk) * (kVs + 2 * kStStride) + (keys > rows ? keys : rows)) * 2;
  if (smem_o > 220 * 1024) return -5;
  if (cudaFuncSetAttribute(linear_chunk_state_kernel<kPair>, cudaFuncAttributeMaxDynamicSharedMemorySize, 80 * 1024) != cudaSuccess ||
      cudaFuncSetAttribute(linear_chunk_out_kernel<kPair, COLS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess)
    return -3;
  launch_pdl(linear_chunk_state_kernel<kPair>, dim3((s.V + 63) / 64, (s.D + 63) / 64, s.H * s.n_req), dim3(128), smem_s, st, a, min_span,
             states);
  launch_pdl(linear_chunk_out_kernel<kPair, COLS>, dim3((s.V + COLS - 1) / COLS, max_chunks, s.H), dim3(256), smem_o, st, a, min_span,
             states);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace stk

using namespace stk;

STK_API long long stk_linear_state_slot(int dim, int vdim) { return linear_slot_floats(dim, vdim); }

// Spans of at least min_span tokens.  q, k: head h's `width` columns at column h / hpg * step of their (already offset) pointers,
// rows ldqk apart; remainders (ql, kl) both or neither.  Either log_decay [heads], the same for every token, or g and w
// [heads, T]: log decay and input weight per token.  skip [heads] or null.  max_chunks bounds the chunks over all requests;
// states: fp32 work space [max_chunks * heads * stk_linear_state_slot()].
STK_API int stk_linear_chunks(const void* qh, const void* ql, const void* kh, const void* kl, long long ldqk, int step, int width, int hpg,
                              const void* v, long long ldv, int v_off, const float* log_decay, const float* g, const float* w,
                              const float* skip, const int* query_start, const int* req_rows, const int* start_pos, int n_req, float* S,
                              float* o, int heads, int dim, int vdim, int min_span, float* states, int max_chunks, int T, void* stream) {
  if (T <= 0 || n_req <= 0 || max_chunks <= 0) return 0;
  if (heads < 1 || dim < 1 || dim > 256 || vdim < 1 || heads > 65535 || static_cast<long long>(heads) * n_req > 65535 ||
      max_chunks > 65535 || min_span < 1 || hpg < 1 || width < dim || (reinterpret_cast<uintptr_t>(states) & 15) ||
      (ql == nullptr) != (kl == nullptr) || (log_decay == nullptr) == (g == nullptr) || (g == nullptr) != (w == nullptr))
    return -1;
  ChunkArgs a;
  a.qh = (const bf16*)qh; a.ql = (const bf16*)ql; a.kh = (const bf16*)kh; a.kl = (const bf16*)kl;
  a.ldqk = ldqk; a.step = step; a.width = width; a.hpg = hpg;
  a.v = (const bf16*)v; a.ldv = ldv; a.v_off = v_off;
  a.fixed = log_decay; a.g = g; a.w = w; a.skip = skip;
  a.s = ScanArgs{query_start, req_rows, start_pos, n_req, S, o, heads, dim, vdim};
  a.T = T;
  cudaStream_t st = (cudaStream_t)stream;
  if (ql != nullptr)
    return vdim <= 64 ? launch_chunks<true, 64>(a, min_span, states, max_chunks, st) : launch_chunks<true, 128>(a, min_span, states, max_chunks, st);
  return vdim <= 64 ? launch_chunks<false, 64>(a, min_span, states, max_chunks, st) : launch_chunks<false, 128>(a, min_span, states, max_chunks, st);
}
