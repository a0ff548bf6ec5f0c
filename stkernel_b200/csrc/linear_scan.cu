// Chunked form of the linear recurrences with a scalar decay (linear_scan.cuh) for bf16 operands: with F the running sum of g inside
// a chunk of 64 tokens and w the tokens' input weights,
//
//   o_t   = exp(F_t) S_start^T q_t + sum_{j <= t} exp(F_t - F_j) w_j (k_j . q_t) v_j  (+ skip v_t)
//   S_end = exp(F_end) S_start + sum_j exp(F_end - F_j) w_j k_j v_j^T
//
//   linear_chunk_state     one CTA per 64 x 64 block of a head's state (transposed: 16 value rows x 32 state rows per warp) walks the chunks of a
//                          request with the block in its accumulators and leaves the state before each chunk
//   linear_chunk_out       per chunk, head and 64 or 128 value columns: the outputs, 16 columns per warp
//
// Both run on the tensor cores.  fp32 operands (weighted values, weighted scores, the state; queries and keys where they come as
// pairs) enter the products as bf16 pairs, high part and remainder, so they keep 16 mantissa bits.  A state is kept as it leaves the
// accumulators: per block of 16 value rows x 16 state rows 32 lanes x 16 bytes of high parts, then of remainders.  An accumulator
// tile of the transposed state has the layout of the B operand that the outputs need, so a lane writes and reads its own 16 bytes.
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
  const float* channel;                          // or, for the states alone, [chunk][H][D] decays of whole chunks per state row
  ScanArgs s;
  int T;
};

// Tokens 2 * lane and 2 * lane + 1 of a chunk of n: running sums of the log decays (F) and input weights (w, 0 behind the chunk).
// One token may decay by thousands and the next ones by thousandths, so sums are formed in fp64 and kept as integer part (x) and
// remainder (y): differences lose nothing.
struct ChunkGates { float2 F0, F1, end; float w0, w1; };
__device__ __forceinline__ float2 int_and_rest(double v) {
  const double i = rint(v);
  return make_float2(static_cast<float>(i), static_cast<float>(v - i));
}
__device__ __forceinline__ float decay_between(float2 later, float2 earlier) { return expf((later.x - earlier.x) + (later.y - earlier.y)); }
struct ChunkRaw { float g0, g1, w0, w1; };

__device__ __forceinline__ ChunkRaw load_gates(const ChunkArgs& a, int h, long long t0, int n, int lane) {
  ChunkRaw r = {0.f, 0.f, 1.f, 1.f};
  if (a.fixed != nullptr) {
    r.g0 = r.g1 = a.fixed[h];
  } else if (a.g != nullptr) {
    const long long at = static_cast<long long>(h) * a.T + t0 + 2 * lane;
    if (2 * lane < n) { r.g0 = a.g[at]; r.w0 = a.w[at]; }
    if (2 * lane + 1 < n) { r.g1 = a.g[at + 1]; r.w1 = a.w[at + 1]; }
  }
  return r;
}
__device__ __forceinline__ ChunkGates chunk_gates(const ChunkArgs& a, const ChunkRaw& r, int n, int lane) {
  ChunkGates c;
  double F0, F1, end;
  if (a.fixed != nullptr) {
    const double g = r.g0;
    F0 = g * (2 * lane + 1);
    F1 = g * (2 * lane + 2);
    end = g * n;
  } else {
    const double pair = static_cast<double>(r.g0) + r.g1;
    double inc = pair;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double up = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += up;
    }
    F0 = inc - r.g1;
    F1 = inc;
    end = __shfl_sync(0xffffffffu, inc, 31);                             // absent tokens add nothing
  }
  c.F0 = int_and_rest(F0);
  c.F1 = int_and_rest(F1);
  c.end = int_and_rest(end);
  c.w0 = 2 * lane < n ? r.w0 : 0.f;
  c.w1 = 2 * lane + 1 < n ? r.w1 : 0.f;
  return c;
}

constexpr int kLsStages = 3;

// kChannel: every state row decays by a factor of its own per chunk, and the keys come with the decays up to the end of their chunk.
template <bool kPair, bool kChannel>
__global__ void __launch_bounds__(256)
linear_chunk_state_kernel(const ChunkArgs a, int min_span, float* __restrict__ states) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  constexpr int kTile = kChunk * kStStride, kParts = kPair ? 2 : 1, kStage = (kParts + 1) * kTile;
  bf16* tiles = reinterpret_cast<bf16*>(smem_raw);                      // [stages]{values, keys (, their remainders)}[64 tokens][72]
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
  const int vw = warp & 3, dw = warp >> 2;                              // the warp's 16 rows, its half of the 64 columns
  const int v0 = vb * 64 + vw * 16 + (lane >> 2), d0 = db * 64 + dw * 32 + (lane & 3) * 2;   // accumulator rows v0 (+ 8), columns d0 + 8 j (+ 1)
  const int nd = blocks16(s.D);
  const long long slot_f = linear_slot_floats(s.D, s.V);
  float* gS = s.S + (row * s.H + h) * static_cast<long long>(s.D) * s.V;
  const int kn = max(0, min(64, a.width - db * 64)), vn = min(64, s.V - vb * 64);
  float acc[4][4];
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int v = v0 + (i >> 1) * 8, d = d0 + j * 8 + (i & 1);
      acc[j][i] = !fresh && d < s.D && v < s.V ? gS[static_cast<long long>(d) * s.V + v] : 0.f;
    }
  const int kc = h / a.hpg * a.step + db * 64;
  auto load = [&](int c) {
    const int n = min(kChunk, span - c * kChunk);
    const long long t0 = q0 + c * kChunk;
    bf16* to = tiles + c % kLsStages * kStage;
    load_rows_async(to, kStStride, 64, a.v + t0 * a.ldv + a.v_off + h * s.V + vb * 64, a.ldv, n, vn, 256);
    load_rows_async(to + kTile, kStStride, 64, a.kh + t0 * a.ldqk + kc, a.ldqk, n, kn, 256);
    if (kPair) load_rows_async(to + 2 * kTile, kStStride, 64, a.kl + t0 * a.ldqk + kc, a.ldqk, n, kn, 256);
  };
  load(0);
  mls_commit();
  if (nc > 1) load(1);
  mls_commit();
  ChunkRaw raw = load_gates(a, h, q0, min(kChunk, span), lane);
  float2 fc[4];                                                       // factors of state columns d0 + 8 j (+ 1)
  auto load_factors = [&](int c) {
    const float* p = a.channel + (static_cast<long long>(first + c) * s.H + h) * s.D;
#pragma unroll
    for (int j = 0; j < 4; ++j) fc[j] = make_float2(d0 + 8 * j < s.D ? p[d0 + 8 * j] : 0.f, d0 + 8 * j + 1 < s.D ? p[d0 + 8 * j + 1] : 0.f);
  };
  if (kChannel) load_factors(0);
  const bool block_ok = vb * 64 + vw * 16 < s.V;                      // warp-uniform: its 16 rows exist
  for (int c = 0; c < nc; ++c) {
    const int n = min(kChunk, span - c * kChunk);
    float w0 = 1.f, w1 = 1.f, fs = 1.f;                                  // weights of tokens 2 lane, 2 lane + 1
    if (!kChannel) {
      const ChunkGates g = chunk_gates(a, raw, n, lane);
      w0 = g.w0 * decay_between(g.end, g.F0);
      w1 = g.w1 * decay_between(g.end, g.F1);
      fs = expf(g.end.x + g.end.y);
    }
    mls_wait<1>();
    __syncthreads();                                                    // chunk c is in, the stage before it is free
    if (c + 2 < nc) load(c + 2);
    mls_commit();
    if (!kChannel && c + 1 < nc) raw = load_gates(a, h, q0 + (c + 1) * kChunk, min(kChunk, span - (c + 1) * kChunk), lane);
    // the state before this chunk
    if (block_ok) {
      float* slot = states + (static_cast<long long>(first + c) * s.H + h) * slot_f +
                    (static_cast<long long>(vb * 4 + vw) * nd + db * 4 + dw * 2) * kBlockFloats;
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        if (db * 4 + dw * 2 + p < nd) {
          uint4 hi, lo;
          mls_split2(acc[2 * p][0], acc[2 * p][1], hi.x, lo.x);
          mls_split2(acc[2 * p + 1][0], acc[2 * p + 1][1], hi.y, lo.y);
          mls_split2(acc[2 * p][2], acc[2 * p][3], hi.z, lo.z);
          mls_split2(acc[2 * p + 1][2], acc[2 * p + 1][3], hi.w, lo.w);
          uint4* to = reinterpret_cast<uint4*>(slot + p * kBlockFloats);
          to[lane] = hi;
          to[32 + lane] = lo;
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[j][i] *= kChannel ? ((i & 1) ? fc[j].y : fc[j].x) : fs;
    if (kChannel && c + 1 < nc) load_factors(c + 1);
    const bf16* v = tiles + c % kLsStages * kStage;
    const bf16* k = v + kTile;
#pragma unroll
    for (int kk = 0; kk < kChunk / 16; ++kk) {
      uint32_t af[4], ah[4], al[4];
      mls_ldsm4_t(af, v + (kk * 16 + (lane & 7) + (lane >> 4) * 8) * kStStride + vw * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int i = 0; i < 2; ++i) {                                     // the operand's token pairs: 2 (lane & 3) and 8 further
        const int from = kk * 8 + i * 4 + (lane & 3);
        const float x0 = __shfl_sync(0xffffffffu, w0, from), x1 = __shfl_sync(0xffffffffu, w1, from);
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&af[2 * i + r]));
          mls_split2(f.x * x0, f.y * x1, ah[2 * i + r], al[2 * i + r]);
        }
      }
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        uint32_t b[4];
        const int off = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kStStride + dw * 32 + j * 16 + (lane >> 4) * 8;
        mls_ldsm4_t(b, k + off);
        mls_mma(acc[2 * j], ah, b[0], b[1]);
        mls_mma(acc[2 * j + 1], ah, b[2], b[3]);
        mls_mma(acc[2 * j], al, b[0], b[1]);
        mls_mma(acc[2 * j + 1], al, b[2], b[3]);
        if (kPair) {
          uint32_t bl[4];
          mls_ldsm4_t(bl, k + kTile + off);
          mls_mma(acc[2 * j], ah, bl[0], bl[1]);
          mls_mma(acc[2 * j + 1], ah, bl[2], bl[3]);
        }
      }
    }
  }
  mls_wait<0>();
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int v = v0 + (i >> 1) * 8, d = d0 + j * 8 + (i & 1);
      if (d < s.D && v < s.V) gS[static_cast<long long>(d) * s.V + v] = acc[j][i];
    }
}

// Row and column of the b-th 16 x 16 block on or below the diagonal.
__device__ __forceinline__ void low_block(int b, int& rb, int& kb) {
  rb = b < 1 ? 0 : b < 3 ? 1 : b < 6 ? 2 : 3;
  kb = b - rb * (rb + 1) / 2;
}

template <bool kPair, int COLS>
__global__ void __launch_bounds__(COLS * 2)
linear_chunk_out_kernel(const ChunkArgs a, int min_span, const float* __restrict__ states) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ float2 s_F[kChunk];
  __shared__ float s_w[kChunk], s_in[kChunk];
  __shared__ ChunkRef s_c;
  __shared__ int s_ok;
  constexpr int kVs = COLS + 8, kParts = kPair ? 2 : 1, kThreads = COLS * 2, kWarps = COLS / 16, kMine = (10 + kWarps - 1) / kWarps;
  const ScanArgs& s = a.s;
  const int Dp = blocks16(s.D) * 16, ks = Dp + 8;
  bf16* q = reinterpret_cast<bf16*>(smem_raw);                          // [parts][64][Dp + 8]
  bf16* v = q + kParts * kChunk * ks;                                   // [64][COLS + 8]
  bf16* k = v + kChunk * kVs;                                           // [parts][64][Dp + 8], then the weighted scores:
  bf16* ph = k;                                                         // [64][72] high parts
  bf16* pl = ph + kChunk * kStStride;                                   // remainders
  pdl_wait();
  pdl_trigger();
  const int vb = blockIdx.x, ci = blockIdx.y, h = blockIdx.z;
  if (threadIdx.x == 0) s_ok = find_chunk(s.query_start, s.n_req, min_span, ci, s_c) ? 1 : 0;
  __syncthreads();
  if (!s_ok) return;
  const ChunkRef c = s_c;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int qc = h / a.hpg * a.step, vn = min(COLS, s.V - vb * COLS);
  // a request's very first chunk starts from zeros: nothing comes from the state
  const bool mine = vb * COLS + warp * 16 < s.V;                        // warp-uniform: its 16 columns exist
  const bool has_state = mine && !(s.start_pos[c.ri] == 0 && c.first == ci);
  const long long at = c.t0 * a.ldqk + qc;
  load_rows_async(q, ks, Dp, a.qh + at, a.ldqk, c.n, a.width, kThreads);
  load_rows_async(k, ks, Dp, a.kh + at, a.ldqk, c.n, a.width, kThreads);
  if (kPair) {
    load_rows_async(q + kChunk * ks, ks, Dp, a.ql + at, a.ldqk, c.n, a.width, kThreads);
    load_rows_async(k + kChunk * ks, ks, Dp, a.kl + at, a.ldqk, c.n, a.width, kThreads);
  }
  load_rows_async(v, kVs, COLS, a.v + c.t0 * a.ldv + a.v_off + h * s.V + vb * COLS, a.ldv, c.n, vn, kThreads);
  mls_commit();
  // this warp's state blocks, a few ahead of the products
  const int nd = Dp / 16;
  constexpr int kAhead = 4;
  const uint4* S = reinterpret_cast<const uint4*>(states + (static_cast<long long>(ci) * s.H + h) * linear_slot_floats(s.D, s.V) +
                                                  static_cast<long long>(vb * kWarps + warp) * nd * kBlockFloats) + lane;
  uint4 sh[kAhead], sl[kAhead];
  if (has_state) {
#pragma unroll
    for (int i = 0; i < kAhead; ++i)
      if (i < nd) {
        sh[i] = __ldcs(S + i * 64);
        sl[i] = __ldcs(S + i * 64 + 32);
      }
  }
  if (warp == 0) {
    const ChunkGates g = chunk_gates(a, load_gates(a, h, c.t0, c.n, lane), c.n, lane);
    s_F[2 * lane] = g.F0;
    s_F[2 * lane + 1] = g.F1;
    s_w[2 * lane] = g.w0;
    s_w[2 * lane + 1] = g.w1;
    s_in[2 * lane] = expf(g.F0.x + g.F0.y);
    s_in[2 * lane + 1] = expf(g.F1.x + g.F1.y);
  }
  mls_wait<0>();
  __syncthreads();
  // weighted scores: the ten blocks on or below the diagonal, in turns over the warps
  uint32_t wh[kMine][4], wl[kMine][4];
#pragma unroll
  for (int m = 0; m < kMine; ++m) {
    const int b = warp + m * kWarps;
    if (b >= 10) continue;
    int rb, kb;
    low_block(b, rb, kb);
    float x[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) x[j][i] = 0.f;
    const int qo = (rb * 16 + (lane & 15)) * ks + (lane >> 4) * 8;
    const int ko = (kb * 16 + (lane >> 4) * 8 + (lane & 7)) * ks + ((lane >> 3) & 1) * 8;
    for (int kk = 0; kk < nd; ++kk) {
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
        const int t = rb * 16 + (lane >> 2) + r * 8, col = kb * 16 + j * 8 + (lane & 3) * 2;
        float p[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) p[i] = col + i <= t ? x[j][2 * r + i] * (s_w[col + i] * decay_between(s_F[t], s_F[col + i])) : 0.f;
        mls_split2(p[0], p[1], wh[m][2 * j + r], wl[m][2 * j + r]);
      }
  }
  __syncthreads();                                                       // the keys are done with
#pragma unroll
  for (int m = 0; m < kMine; ++m) {
    const int b = warp + m * kWarps;
    if (b >= 10) continue;
    int rb, kb;
    low_block(b, rb, kb);
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int off = (rb * 16 + (lane >> 2) + r * 8) * kStStride + kb * 16 + j * 8 + (lane & 3) * 2;
        *reinterpret_cast<uint32_t*>(ph + off) = wh[m][2 * j + r];
        *reinterpret_cast<uint32_t*>(pl + off) = wl[m][2 * j + r];
      }
  }
  float o[4][2][4];
#pragma unroll
  for (int rb = 0; rb < 4; ++rb)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) o[rb][j][i] = 0.f;
  if (has_state) {
    const bf16* qa = q + (lane & 15) * ks + (lane >> 4) * 8;
    for (int k0 = 0; k0 < nd; k0 += kAhead) {
#pragma unroll
      for (int i = 0; i < kAhead; ++i) {
        const int kk = k0 + i;
        if (kk >= nd) continue;
        const uint4 hi = sh[i], lo = sl[i];
        if (kk + kAhead < nd) {
          sh[i] = __ldcs(S + (kk + kAhead) * 64);
          sl[i] = __ldcs(S + (kk + kAhead) * 64 + 32);
        }
#pragma unroll
        for (int rb = 0; rb < 4; ++rb) {
          uint32_t af[4];
          mls_ldsm4(af, qa + rb * 16 * ks + kk * 16);
          mls_mma(o[rb][0], af, hi.x, hi.y);
          mls_mma(o[rb][1], af, hi.z, hi.w);
          mls_mma(o[rb][0], af, lo.x, lo.y);
          mls_mma(o[rb][1], af, lo.z, lo.w);
          if (kPair) {
            uint32_t al[4];
            mls_ldsm4(al, qa + (kChunk + rb * 16) * ks + kk * 16);
            mls_mma(o[rb][0], al, hi.x, hi.y);
            mls_mma(o[rb][1], al, hi.z, hi.w);
          }
        }
      }
    }
#pragma unroll
    for (int rb = 0; rb < 4; ++rb)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float f = s_in[rb * 16 + (lane >> 2) + (i >> 1) * 8];
        o[rb][0][i] *= f;
        o[rb][1][i] *= f;
      }
  }
  __syncthreads();                                                       // the weighted scores are complete
  if (!mine) return;
#pragma unroll
  for (int kb = 0; kb < 4; ++kb) {
    uint32_t b[4];
    mls_ldsm4_t(b, v + (kb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kVs + warp * 16 + (lane >> 4) * 8);
#pragma unroll
    for (int rb = kb; rb < 4; ++rb) {
      uint32_t hi[4], lo[4];
      const int off = (rb * 16 + (lane & 15)) * kStStride + kb * 16 + (lane >> 4) * 8;
      mls_ldsm4(hi, ph + off);
      mls_ldsm4(lo, pl + off);
      mls_mma(o[rb][0], hi, b[0], b[1]);
      mls_mma(o[rb][1], hi, b[2], b[3]);
      mls_mma(o[rb][0], lo, b[0], b[1]);
      mls_mma(o[rb][1], lo, b[2], b[3]);
    }
  }
  const float skip = a.skip != nullptr ? a.skip[h] : 0.f;
  const bool pair = (s.V & 1) == 0;
#pragma unroll
  for (int rb = 0; rb < 4; ++rb)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = rb * 16 + (lane >> 2) + r * 8;
      if (t >= c.n) continue;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int lc = warp * 16 + j * 8 + (lane & 3) * 2, col = vb * COLS + lc;
        const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v + t * kVs + lc));
        const float y0 = fmaf(skip, x.x, o[rb][j][2 * r]), y1 = fmaf(skip, x.y, o[rb][j][2 * r + 1]);
        float* out = s.o + ((c.t0 + t) * static_cast<long long>(s.H) + h) * s.V + col;
        if (pair && col + 1 < s.V) {
          *reinterpret_cast<float2*>(out) = make_float2(y0, y1);
        } else {
          if (col < s.V) out[0] = y0;
          if (col + 1 < s.V) out[1] = y1;
        }
      }
    }
}

template <bool kPair, int COLS>
static int launch_chunks(const ChunkArgs& a, int min_span, float* states, int max_chunks, cudaStream_t st) {
  constexpr int kParts = kPair ? 2 : 1, kVs = COLS + 8;
  const ScanArgs& s = a.s;
  const int ks = blocks16(s.D) * 16 + 8;
  const size_t smem_s = static_cast<size_t>(kLsStages) * (kParts + 1) * kChunk * kStStride * 2;
  const size_t keys = static_cast<size_t>(kParts) * kChunk * ks, scores = static_cast<size_t>(2) * kChunk * kStStride;
  const size_t smem_o = (keys + static_cast<size_t>(kChunk) * kVs + (keys > scores ? keys : scores)) * 2;
  if (smem_o > 220 * 1024) return -5;
  if (cudaFuncSetAttribute(linear_chunk_state_kernel<kPair, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 84 * 1024) != cudaSuccess ||
      cudaFuncSetAttribute(linear_chunk_out_kernel<kPair, COLS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess)
    return -3;
  launch_pdl(linear_chunk_state_kernel<kPair, false>, dim3((s.V + 63) / 64, (s.D + 63) / 64, s.H * s.n_req), dim3(256), smem_s, st, a, min_span,
             states);
  launch_pdl(linear_chunk_out_kernel<kPair, COLS>, dim3((s.V + COLS - 1) / COLS, max_chunks, s.H), dim3(COLS * 2), smem_o, st, a, min_span,
             states);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

int linear_states_per_channel(const bf16* kh, const bf16* kl, long long ldk, int step, int width, const bf16* v, long long ldv, int v_off,
                              const float* channel, const ScanArgs& s, int min_span, float* states, int T, cudaStream_t st) {
  ChunkArgs a = {};
  a.kh = kh; a.kl = kl; a.ldqk = ldk; a.step = step; a.width = width; a.hpg = 1;
  a.v = v; a.ldv = ldv; a.v_off = v_off; a.channel = channel; a.s = s; a.T = T;
  const size_t smem = static_cast<size_t>(kLsStages) * 3 * kChunk * kStStride * 2;
  if (cudaFuncSetAttribute(linear_chunk_state_kernel<true, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 84 * 1024) != cudaSuccess)
    return -3;
  launch_pdl(linear_chunk_state_kernel<true, true>, dim3((s.V + 63) / 64, (s.D + 63) / 64, s.H * s.n_req), dim3(256), smem, st, a, min_span,
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
  a.fixed = log_decay; a.g = g; a.w = w; a.skip = skip; a.channel = nullptr;
  a.s = ScanArgs{query_start, req_rows, start_pos, n_req, S, o, heads, dim, vdim};
  a.T = T;
  cudaStream_t st = (cudaStream_t)stream;
  if (ql != nullptr)
    return vdim <= 64 ? launch_chunks<true, 64>(a, min_span, states, max_chunks, st) : launch_chunks<true, 128>(a, min_span, states, max_chunks, st);
  return vdim <= 64 ? launch_chunks<false, 64>(a, min_span, states, max_chunks, st) : launch_chunks<false, 128>(a, min_span, states, max_chunks, st);
}
