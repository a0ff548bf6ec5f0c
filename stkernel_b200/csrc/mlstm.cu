// mLSTM: matrix-memory recurrence with exponential input gate, forget gate and running-maximum stabiliser.
//
//   m_t = max(f_t + m_{t-1}, i_t)
//   S_t = exp(f_t + m_{t-1} - m_t) S_{t-1} + exp(i_t - m_t) k_t v_t^T        n_t likewise with k_t alone
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
//
// Every kernel here leaves the numerator S_t^T q_t, the normaliser n_t . q_t and m_t of each token in fp32; mlstm_finish
// divides, norms each head, applies the output gate and advances the stored maximum (so kernels that run over disjoint
// column blocks of a head all read the same m_{t-1}).  A span that starts at position 0 starts from a zero state.
//
//   mlstm_scan          token by token, any size and type: one CTA per (32 value columns, head, request), state in shared memory
//   mlstm_chunk_*       prompt portions, bf16 operands: with F the running sum of f inside a chunk of 64 tokens, a_j = i_j - F_j
//                       and M_t = max(m_start, max_{j<=t} a_j), the recurrence is
//                         m_t = F_t + M_t,  S_t^T q_t = exp(m_start - M_t) S_start^T q_t + sum_{j<=t} exp(a_j - M_t) (k_j . q_t) v_j
//                       (1) gates: the records a, F and the chain of m over the chunks;  (2) states: one CTA per 64 x 64 block of
//                       a head's memory walks the chunks with the block in its accumulators and leaves the state before each
//                       chunk as bf16 pairs (high part and remainder);  (3) per chunk: the outputs.  (2) and (3) run on the
//                       tensor cores with the fp32 operand of each product as a bf16 pair (16 mantissa bits).
// Sums of log gates reach hundreds, so they are formed in fp64 and kept as integer part + remainder: differences lose nothing.
#define STK_PDL_CLASS 16
#include "chunk_mma.cuh"
#include "hybrid_block.cuh"

namespace stk {

constexpr int kGateSlot = 3 * kChunk + 8;      // a (integer, remainder), F; A, F_end, m_start, M_end as (integer, remainder) pairs

struct MlstmArgs {
  const void* proj; long long ldp; int q_off, k_off, v_off;
  const float* gates; const float* gate_bias; float cap;
  const int* query_start; const int* req_rows; const int* start_pos; int n_req;
  float* S; float* n; float* m;
  float* num; float* den; float* mt;
  int H, D, V;
};

__device__ __forceinline__ float ml_f(float v) { return v; }
__device__ __forceinline__ float ml_f(__nv_bfloat16 v) { return bf16_to_f(v); }

__device__ __forceinline__ void log_gates(const MlstmArgs& a, long long t, int h, float& ig, float& fg) {
  const float* g = a.gates + t * 2 * a.H;
  ig = a.cap * tanhf((g[h] + a.gate_bias[h]) / a.cap);
  const float x = a.cap * tanhf((g[a.H + h] + a.gate_bias[a.H + h]) / a.cap);
  fg = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}

// ---- token by token ---------------------------------------------------------------------------------
constexpr int kScanCols = 32;

template <typename A>
__global__ void __launch_bounds__(256)
mlstm_scan_kernel(const MlstmArgs a, int min_span, int max_span) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  float* S = sm;                                  // [D][32]
  float* nn = S + a.D * kScanCols;                // [D]
  float* q = nn + a.D;                            // [D]
  float* k = q + a.D;                             // [D]
  float* part = k + a.D;                          // [8][32]
  pdl_wait();
  pdl_trigger();
  const int vb = blockIdx.x, h = blockIdx.y, ri = blockIdx.z;
  const int q0 = a.query_start[ri], span = a.query_start[ri + 1] - q0;
  if (span <= 0 || span < min_span || span > max_span) return;
  const long long row = a.req_rows[ri];
  const bool fresh = a.start_pos[ri] == 0;
  const int c = threadIdx.x & 31, r = threadIdx.x >> 5;
  const int col = vb * kScanCols + c;
  const bool col_ok = col < a.V;
  float* gS = a.S + (row * a.H + h) * a.D * a.V;
  float* gn = a.n + (row * a.H + h) * a.D;
  for (int d = r; d < a.D; d += 8) S[d * kScanCols + c] = col_ok && !fresh ? gS[static_cast<long long>(d) * a.V + col] : 0.f;
  if (vb == 0)
    for (int d = threadIdx.x; d < a.D; d += 256) nn[d] = fresh ? 0.f : gn[d];
  float m = fresh ? 0.f : a.m[row * a.H + h];
  const float qs = 1.f / sqrtf(static_cast<float>(a.D));
  for (int i = 0; i < span; ++i) {
    const long long t = q0 + i;
    const A* p = reinterpret_cast<const A*>(a.proj) + t * a.ldp;
    __syncthreads();
    for (int d = threadIdx.x; d < a.D; d += 256) {
      q[d] = ml_f(p[a.q_off + h * a.D + d]) * qs;
      k[d] = ml_f(p[a.k_off + h * a.D + d]);
    }
    const float v = col_ok ? ml_f(p[a.v_off + h * a.V + col]) : 0.f;
    float ig, fg;
    log_gates(a, t, h, ig, fg);
    const float m_new = fmaxf(fg + m, ig);
    const float fa = expf(fg + m - m_new), fb = expf(ig - m_new);
    m = m_new;
    __syncthreads();
    float acc = 0.f;
    const float bv = fb * v;
    for (int d = r; d < a.D; d += 8) {
      const float s = fmaf(fa, S[d * kScanCols + c], k[d] * bv);
      S[d * kScanCols + c] = s;
      acc = fmaf(q[d], s, acc);
    }
    part[r * kScanCols + c] = acc;
    if (vb == 0) {
      float nq = 0.f;
      for (int d = threadIdx.x; d < a.D; d += 256) {
        const float x = fmaf(fa, nn[d], fb * k[d]);
        nn[d] = x;
        nq = fmaf(q[d], x, nq);
      }
      nq = block_sum(nq, red);
      if (threadIdx.x == 0) {
        a.den[t * a.H + h] = nq;
        a.mt[t * a.H + h] = m;
      }
    } else {
      __syncthreads();
    }
    if (r == 0 && col_ok) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) s += part[w * kScanCols + c];
      a.num[(t * a.H + h) * a.V + col] = s;
    }
  }
  __syncthreads();
  if (col_ok)
    for (int d = r; d < a.D; d += 8) gS[static_cast<long long>(d) * a.V + col] = S[d * kScanCols + c];
  if (vb == 0)
    for (int d = threadIdx.x; d < a.D; d += 256) gn[d] = nn[d];
}

// ---- chunks -------------------------------------------------------------------------------------------
// A chunk's state before its first token: [D][Vp] high parts, [D][Vp] remainders (bf16), then n[D] fp32; Vp = V rounded up to 8.
// Slots are whole 16-byte units.
__host__ __device__ inline long long state_slot_floats(int D, int V) {
  return (static_cast<long long>(D) * ((V + 7) / 8 * 8 + 1) + 3) / 4 * 4;
}

// (1) gate records of every chunk of one (head, request), then the chain of running maxima over its chunks.
__global__ void __launch_bounds__(256)
mlstm_chunk_gates_kernel(const MlstmArgs a, int min_span, float* __restrict__ gate_ws) {
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, ri = blockIdx.y;
  const int q0 = a.query_start[ri], span = a.query_start[ri + 1] - q0;
  if (span < min_span || span <= 0) return;
  const int first = first_chunk(a.query_start, min_span, ri), nc = (span + kChunk - 1) / kChunk;
  const int warp = threadIdx.x >> 5, l = threadIdx.x & 31;
  for (int c = warp; c < nc; c += 8) {
    const int t0 = q0 + c * kChunk, n = min(kChunk, span - c * kChunk);
    float i0 = 0.f, i1 = 0.f, g0 = 0.f, g1 = 0.f;
    if (2 * l < n) log_gates(a, t0 + 2 * l, h, i0, g0);
    if (2 * l + 1 < n) log_gates(a, t0 + 2 * l + 1, h, i1, g1);
    // running sum of the log forget gates over 64 tokens, two per lane
    const double f0 = g0, pair = f0 + g1;
    double inc = pair;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double up = __shfl_up_sync(0xffffffffu, inc, o);
      if (l >= o) inc += up;
    }
    const double F0 = inc - pair + f0, F1 = inc;                    // absent tokens add nothing
    const double a0 = 2 * l < n ? i0 - F0 : -1e30, a1 = 2 * l + 1 < n ? i1 - F1 : -1e30;
    double mx = a0 > a1 ? a0 : a1;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const double other = __shfl_xor_sync(0xffffffffu, mx, o);
      mx = other > mx ? other : mx;
    }
    const double fe = __shfl_sync(0xffffffffu, inc, 31);
    float* g = gate_ws + (static_cast<long long>(first + c) * a.H + h) * kGateSlot;
    const double r0 = rint(a0), r1 = rint(a1);
    g[2 * l] = static_cast<float>(r0);
    g[2 * l + 1] = static_cast<float>(r1);
    g[kChunk + 2 * l] = static_cast<float>(a0 - r0);
    g[kChunk + 2 * l + 1] = static_cast<float>(a1 - r1);
    g[2 * kChunk + 2 * l] = static_cast<float>(F0);
    g[2 * kChunk + 2 * l + 1] = static_cast<float>(F1);
    if (l == 0) {
      const double ai = rint(mx), fi = rint(fe);
      g[3 * kChunk + 0] = static_cast<float>(ai);
      g[3 * kChunk + 1] = static_cast<float>(mx - ai);
      g[3 * kChunk + 2] = static_cast<float>(fi);
      g[3 * kChunk + 3] = static_cast<float>(fe - fi);
    }
  }
  __syncthreads();
  if (warp != 0) return;
  double m = a.start_pos[ri] == 0 ? 0.0 : static_cast<double>(a.m[static_cast<long long>(a.req_rows[ri]) * a.H + h]);
  for (int base = 0; base < nc; base += 32) {
    const int c = base + l;
    float* g = gate_ws + (static_cast<long long>(first + c) * a.H + h) * kGateSlot + 3 * kChunk;
    double A = 0.0, F = 0.0, mine = 0.0, top = 0.0;
    if (c < nc) {
      A = static_cast<double>(g[0]) + g[1];
      F = static_cast<double>(g[2]) + g[3];
    }
    const int cnt = min(32, nc - base);
    for (int i = 0; i < cnt; ++i) {
      const double Ai = __shfl_sync(0xffffffffu, A, i), Fi = __shfl_sync(0xffffffffu, F, i);
      const double M = m > Ai ? m : Ai;
      if (l == i) { mine = m; top = M; }
      m = Fi + M;
    }
    if (c < nc) {
      const double mi = rint(mine), ti = rint(top);
      g[4] = static_cast<float>(mi);
      g[5] = static_cast<float>(mine - mi);
      g[6] = static_cast<float>(ti);
      g[7] = static_cast<float>(top - ti);
    }
  }
}

// (2) states.  One CTA: 64 memory rows x 64 value columns of one head of one request, all its chunks in order.
__global__ void __launch_bounds__(128)
mlstm_chunk_state_kernel(const MlstmArgs a, int min_span, const float* __restrict__ gate_ws, float* __restrict__ states) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ float s_w[kChunk];
  __shared__ float s_fs;
  constexpr int kTile = kChunk * kStStride;
  __nv_bfloat16* kt = reinterpret_cast<__nv_bfloat16*>(smem_raw);       // two stages of [64 tokens][72]
  __nv_bfloat16* vt = kt + 2 * kTile;
  __nv_bfloat16* vh = vt + 2 * kTile;                                   // weighted values, high part
  __nv_bfloat16* vl = vh + kTile;                                       // remainder
  pdl_wait();
  pdl_trigger();
  const int vb = blockIdx.x, db = blockIdx.y, h = blockIdx.z % a.H, ri = blockIdx.z / a.H;
  const int q0 = a.query_start[ri], span = a.query_start[ri + 1] - q0;
  if (span < min_span || span <= 0) return;
  const int first = first_chunk(a.query_start, min_span, ri), nc = (span + kChunk - 1) / kChunk;
  const long long row = a.req_rows[ri];
  const bool fresh = a.start_pos[ri] == 0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int d0 = db * 64 + warp * 16 + (lane >> 2), c0 = vb * 64 + (lane & 3) * 2;
  const int Vp = (a.V + 7) / 8 * 8;
  const long long slot_f = state_slot_floats(a.D, a.V);
  float* gS = a.S + (row * a.H + h) * static_cast<long long>(a.D) * a.V;
  float* gn = a.n + (row * a.H + h) * a.D;
  const int dn = min(64, a.D - db * 64), vn = min(64, a.V - vb * 64);
  float acc[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = d0 + (i >> 1) * 8, c = c0 + j * 8 + (i & 1);
      acc[j][i] = !fresh && d < a.D && c < a.V ? gS[static_cast<long long>(d) * a.V + c] : 0.f;
    }
  // normaliser of this CTA's rows (first column block): one thread per row in the first two warps
  const int nd = threadIdx.x & 63, nh = threadIdx.x >> 6;
  float nacc = vb == 0 && nh == 0 && nd < dn && !fresh ? gn[db * 64 + nd] : 0.f;
  const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(a.proj);
  auto load = [&](int c) {
    const int n = min(kChunk, span - c * kChunk), st = c & 1;
    const __nv_bfloat16* p = proj + static_cast<long long>(q0 + c * kChunk) * a.ldp;
    load_rows_async(kt + st * kTile, kStStride, 64, p + a.k_off + h * a.D + db * 64, a.ldp, n, dn, 128);
    load_rows_async(vt + st * kTile, kStStride, 64, p + a.v_off + h * a.V + vb * 64, a.ldp, n, vn, 128);
  };
  float w_next = 0.f, fs_next = 0.f;
  auto gates = [&](int c) {
    const float* g = gate_ws + (static_cast<long long>(first + c) * a.H + h) * kGateSlot;
    const float ti = g[3 * kChunk + 6], tr = g[3 * kChunk + 7];
    if (threadIdx.x < kChunk) w_next = expf((g[threadIdx.x] - ti) + (g[kChunk + threadIdx.x] - tr));
    if (threadIdx.x == kChunk) fs_next = expf((g[3 * kChunk + 4] - ti) + (g[3 * kChunk + 5] - tr));
  };
  load(0);
  mls_commit();
  gates(0);
  for (int c = 0; c < nc; ++c) {
    if (threadIdx.x < kChunk) s_w[threadIdx.x] = w_next;
    if (threadIdx.x == kChunk) s_fs = fs_next;
    if (c + 1 < nc) load(c + 1);
    mls_commit();
    mls_wait<1>();
    __syncthreads();
    if (c + 1 < nc) gates(c + 1);
    // the state before this chunk
    {
      float* slot = states + (static_cast<long long>(first + c) * a.H + h) * slot_f;
      __nv_bfloat16* sh = reinterpret_cast<__nv_bfloat16*>(slot);
      __nv_bfloat16* sl = sh + static_cast<long long>(a.D) * Vp;
#pragma unroll
      for (int j = 0; j < 8; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int d = d0 + r * 8, col = c0 + j * 8;
          if (d < a.D && col < Vp) {
            uint32_t hi, lo;
            mls_split2(acc[j][2 * r], acc[j][2 * r + 1], hi, lo);
            *reinterpret_cast<uint32_t*>(sh + static_cast<long long>(d) * Vp + col) = hi;
            *reinterpret_cast<uint32_t*>(sl + static_cast<long long>(d) * Vp + col) = lo;
          }
        }
      if (vb == 0 && nh == 0 && nd < dn) slot[static_cast<long long>(a.D) * Vp + db * 64 + nd] = nacc;
    }
    const __nv_bfloat16* k = kt + (c & 1) * kTile;
    const __nv_bfloat16* v = vt + (c & 1) * kTile;
    for (int e = threadIdx.x; e < kChunk * 32; e += 128) {
      const int r = e >> 5, cc = (e & 31) * 2;
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(v + r * kStStride + cc));
      const float w = s_w[r];
      uint32_t hi, lo;
      mls_split2(x.x * w, x.y * w, hi, lo);
      *reinterpret_cast<uint32_t*>(vh + r * kStStride + cc) = hi;
      *reinterpret_cast<uint32_t*>(vl + r * kStStride + cc) = lo;
    }
    const float fs = s_fs;
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[j][i] *= fs;
    if (vb == 0 && nh == 0) {
      float s = 0.f, s2 = 0.f;
#pragma unroll 8
      for (int t = 0; t < kChunk; t += 2) {
        s = fmaf(s_w[t], bf16_to_f(k[t * kStStride + nd]), s);
        s2 = fmaf(s_w[t + 1], bf16_to_f(k[(t + 1) * kStStride + nd]), s2);
      }
      nacc = fmaf(fs, nacc, s + s2);
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < kChunk / 16; ++kk) {
      uint32_t af[4];
      mls_ldsm4_t(af, k + (kk * 16 + (lane & 7) + (lane >> 4) * 8) * kStStride + warp * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        uint32_t bh[4], bl[4];
        const int off = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kStStride + j * 16 + (lane >> 4) * 8;
        mls_ldsm4_t(bh, vh + off);
        mls_ldsm4_t(bl, vl + off);
        mls_mma(acc[2 * j], af, bh[0], bh[1]);
        mls_mma(acc[2 * j + 1], af, bh[2], bh[3]);
        mls_mma(acc[2 * j], af, bl[0], bl[1]);
        mls_mma(acc[2 * j + 1], af, bl[2], bl[3]);
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
      if (d < a.D && c < a.V) gS[static_cast<long long>(d) * a.V + c] = acc[j][i];
    }
  if (vb == 0 && nh == 0 && nd < dn) gn[db * 64 + nd] = nacc;
}

// (3) outputs of a chunk for 128 value columns; the first column block also writes n_t . q_t and m_t.  Eight warps: four
// blocks of 16 tokens x two halves of the columns (of the keys while the scores are formed).
constexpr int kOutCols = 128, kOutStride = kOutCols + 8, kOutRows = 32;

__global__ void __launch_bounds__(256)
mlstm_chunk_out_kernel(const MlstmArgs a, int min_span, const float* __restrict__ gate_ws, const float* __restrict__ states) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ float s_ai[kChunk], s_ar[kChunk], s_mi[kChunk], s_mr[kChunk], s_in[kChunk], s_nq[kChunk], s_sum[2][kChunk];
  __shared__ ChunkRef s_c;
  __shared__ int s_ok;
  const int Dp = (a.D + 15) / 16 * 16, ks = Dp + 8;
  __nv_bfloat16* q = reinterpret_cast<__nv_bfloat16*>(smem_raw);        // [64][Dp + 8]
  __nv_bfloat16* v = q + kChunk * ks;                                   // [64][136]
  __nv_bfloat16* ph = v + kChunk * kOutStride;                          // [64][72] weighted scores, high part
  __nv_bfloat16* pl = ph + kChunk * kStStride;                          // remainder
  __nv_bfloat16* k = pl + kChunk * kStStride;                           // [64][Dp + 8], then two stages of state rows:
  __nv_bfloat16* st = k;                                                // {high, remainder} x [32][136]
  pdl_wait();
  pdl_trigger();
  const int vb = blockIdx.x, ci = blockIdx.y, h = blockIdx.z;
  if (threadIdx.x == 0) s_ok = find_chunk(a.query_start, a.n_req, min_span, ci, s_c) ? 1 : 0;
  __syncthreads();
  if (!s_ok) return;
  const ChunkRef c = s_c;
  const __nv_bfloat16* p = reinterpret_cast<const __nv_bfloat16*>(a.proj) + c.t0 * a.ldp;
  const long long slot = static_cast<long long>(ci) * a.H + h;
  const float* g = gate_ws + slot * kGateSlot;
  const int Vp = (a.V + 7) / 8 * 8;
  const float* base = states + slot * state_slot_floats(a.D, a.V);
  const __nv_bfloat16* Sh = reinterpret_cast<const __nv_bfloat16*>(base);
  const __nv_bfloat16* Sl = Sh + static_cast<long long>(a.D) * Vp;
  const float* n0 = base + static_cast<long long>(a.D) * Vp;
  // a request's very first chunk starts from zeros: nothing comes from the state
  const bool has_state = !(a.start_pos[c.ri] == 0 && c.first == ci);
  load_rows_async(q, ks, Dp, p + a.q_off + h * a.D, a.ldp, c.n, a.D, 256);
  load_rows_async(k, ks, Dp, p + a.k_off + h * a.D, a.ldp, c.n, a.D, 256);
  load_rows_async(v, kOutStride, kOutCols, p + a.v_off + h * a.V + vb * kOutCols, a.ldp, c.n, min(kOutCols, a.V - vb * kOutCols), 256);
  mls_commit();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rb = warp & 3, half = warp >> 2;
  if (warp == 0) {
    // M_t = max(m_start, running max of a), two tokens per lane
    const double m0 = static_cast<double>(g[3 * kChunk + 4]) + g[3 * kChunk + 5];
    const double a0 = static_cast<double>(g[2 * lane]) + g[kChunk + 2 * lane];
    const double a1 = static_cast<double>(g[2 * lane + 1]) + g[kChunk + 2 * lane + 1];
    double inc = a0 > a1 ? a0 : a1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double up = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o && up > inc) inc = up;
    }
    double before = __shfl_up_sync(0xffffffffu, inc, 1);
    if (lane == 0 || before < m0) before = m0;
    const double M0 = before > a0 ? before : a0, M1 = M0 > a1 ? M0 : a1;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int j = 2 * lane + i;
      const double M = i == 0 ? M0 : M1, mi = rint(M);
      s_ai[j] = g[j];
      s_ar[j] = g[kChunk + j];
      s_mi[j] = static_cast<float>(mi);
      s_mr[j] = static_cast<float>(M - mi);
      s_in[j] = expf(static_cast<float>(m0 - M));
      if (vb == 0 && j < c.n) a.mt[(c.t0 + j) * static_cast<long long>(a.H) + h] = static_cast<float>(g[2 * kChunk + j] + M);
    }
  }
  mls_wait<0>();
  __syncthreads();
  const float qs = 1.f / sqrtf(static_cast<float>(a.D));
  int row[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) row[r] = rb * 16 + (lane >> 2) + r * 8;
  // weighted scores of this warp's tokens against every other block of 16 keys
  {
    float sum[2] = {0.f, 0.f};
    const float mi[2] = {s_mi[row[0]], s_mi[row[1]]}, mr[2] = {s_mr[row[0]], s_mr[row[1]]};
    for (int kb = half; kb <= rb; kb += 2) {
      float s[2][4];
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) s[j][i] = 0.f;
      for (int kk = 0; kk < Dp / 16; ++kk) {
        uint32_t af[4], bf[4];
        mls_ldsm4(af, q + (rb * 16 + (lane & 15)) * ks + kk * 16 + (lane >> 4) * 8);
        mls_ldsm4(bf, k + (kb * 16 + (lane >> 4) * 8 + (lane & 7)) * ks + kk * 16 + ((lane >> 3) & 1) * 8);
        mls_mma(s[0], af, bf[0], bf[1]);
        mls_mma(s[1], af, bf[2], bf[3]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int col = kb * 16 + j * 8 + (lane & 3) * 2;
          float x[2];
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const float w = col + i <= row[r] ? expf((s_ai[col + i] - mi[r]) + (s_ar[col + i] - mr[r])) : 0.f;
            x[i] = s[j][2 * r + i] * w;
            sum[r] += x[i];
          }
          uint32_t hi, lo;
          mls_split2(x[0], x[1], hi, lo);
          *reinterpret_cast<uint32_t*>(ph + row[r] * kStStride + col) = hi;
          *reinterpret_cast<uint32_t*>(pl + row[r] * kStStride + col) = lo;
        }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
      sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
      if ((lane & 3) == 0) s_sum[half][row[r]] = sum[r];
    }
  }
  if (vb == 0) {
    for (int r = warp * 8; r < warp * 8 + 8; ++r) {
      float s = 0.f;
      if (has_state)
        for (int d = lane; d < a.D; d += 32) s = fmaf(bf16_to_f(q[r * ks + d]), n0[d], s);
      s = warp_sum(s);
      if (lane == 0) s_nq[r] = s;
    }
  }
  __syncthreads();                                                       // k is free, the weighted scores are complete
  float o[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[j][i] = 0.f;
  if (has_state) {
    const int slices = (Dp + kOutRows - 1) / kOutRows, ch = kOutCols / 8;
    auto load_slice = [&](int sl) {
      __nv_bfloat16* dst = st + (sl & 1) * 2 * kOutRows * kOutStride;
      for (int e = threadIdx.x; e < 2 * kOutRows * ch; e += 256) {
        const int part = e / (kOutRows * ch), r = e / ch % kOutRows, cc = e % ch * 8;
        const int d = sl * kOutRows + r, col = vb * kOutCols + cc;
        const bool ok = d < a.D && col < Vp;
        const __nv_bfloat16* src = (part ? Sl : Sh) + (ok ? static_cast<long long>(d) * Vp + col : 0);
        mls_cp16(dst + (part * kOutRows + r) * kOutStride + cc, src, ok);
      }
    };
    load_slice(0);
    mls_commit();
    for (int sl = 0; sl < slices; ++sl) {
      if (sl + 1 < slices) load_slice(sl + 1);
      mls_commit();
      mls_wait<1>();
      __syncthreads();
      const __nv_bfloat16* hi = st + (sl & 1) * 2 * kOutRows * kOutStride;
      const __nv_bfloat16* lo = hi + kOutRows * kOutStride;
#pragma unroll
      for (int kk = 0; kk < kOutRows / 16; ++kk) {
        if (sl * kOutRows + kk * 16 < Dp) {
          uint32_t af[4];
          mls_ldsm4(af, q + (rb * 16 + (lane & 15)) * ks + sl * kOutRows + kk * 16 + (lane >> 4) * 8);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            uint32_t bh[4], bl[4];
            const int off = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kOutStride + half * 64 + j * 16 + (lane >> 4) * 8;
            mls_ldsm4_t(bh, hi + off);
            mls_ldsm4_t(bl, lo + off);
            mls_mma(o[2 * j], af, bh[0], bh[1]);
            mls_mma(o[2 * j + 1], af, bh[2], bh[3]);
            mls_mma(o[2 * j], af, bl[0], bl[1]);
            mls_mma(o[2 * j + 1], af, bl[2], bl[3]);
          }
        }
      }
      __syncthreads();
    }
    mls_wait<0>();
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) o[j][i] *= s_in[row[i >> 1]];
  }
  for (int kb = 0; kb <= rb; ++kb) {
    uint32_t hi[4], lo[4];
    const int off = (rb * 16 + (lane & 15)) * kStStride + kb * 16 + (lane >> 4) * 8;
    mls_ldsm4(hi, ph + off);
    mls_ldsm4(lo, pl + off);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      uint32_t bf[4];
      mls_ldsm4_t(bf, v + (kb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * kOutStride + half * 64 + j * 16 + (lane >> 4) * 8);
      mls_mma(o[2 * j], hi, bf[0], bf[1]);
      mls_mma(o[2 * j + 1], hi, bf[2], bf[3]);
      mls_mma(o[2 * j], lo, bf[0], bf[1]);
      mls_mma(o[2 * j + 1], lo, bf[2], bf[3]);
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    if (row[r] >= c.n) continue;
    const long long t = c.t0 + row[r];
    if (vb == 0 && half == 0 && (lane & 3) == 0)
      a.den[t * a.H + h] = (s_sum[0][row[r]] + s_sum[1][row[r]] + s_in[row[r]] * s_nq[row[r]]) * qs;
    const int c0 = vb * kOutCols + half * 64 + (lane & 3) * 2;
    float* out = a.num + (t * a.H + h) * a.V + c0;
    const bool pair = (a.V & 1) == 0;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float x = o[j][2 * r] * qs, y = o[j][2 * r + 1] * qs;
      if (pair && c0 + j * 8 + 1 < a.V) {
        *reinterpret_cast<float2*>(out + j * 8) = make_float2(x, y);
      } else {
        if (c0 + j * 8 < a.V) out[j * 8] = x;
        if (c0 + j * 8 + 1 < a.V) out[j * 8 + 1] = y;
      }
    }
  }
}

// ---- head norm, output gate, stored maximum, feed-forward activation -----------------------------------
// out[t, h * V + c] = o / rms(o over the head) * w * sigmoid(g), o = num / (max(|den|, exp(-m)) + 1e-6): one warp per (token,
// head) in the first `head_blocks` blocks; the blocks after them form the feed-forward half, 2048 columns of a token each.
template <typename A>
__global__ void __launch_bounds__(256)
mlstm_finish_kernel(const float* __restrict__ num, const float* __restrict__ den, const float* __restrict__ mt,
                    float* __restrict__ m_state, const float* __restrict__ w, float eps, const int* __restrict__ tok_req,
                    const int64_t* __restrict__ positions, const int* __restrict__ last_pos, const A* __restrict__ proj,
                    long long ldp, int g_off, A* __restrict__ out, long long ldo, int H, int V, int go, int uo, int ff, int o0,
                    int cols, int T, int head_blocks, int ff_blocks) {
  pdl_wait();
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (static_cast<int>(blockIdx.x) >= head_blocks) {
    const int b = blockIdx.x - head_blocks;
    const long long t = b / ff_blocks;
    const A* p = proj + t * ldp;
    A* o = out + t * ldo;
    glu_columns(p + go, p + uo, o + o0, (b % ff_blocks * 256 + static_cast<int>(threadIdx.x)) * 8, ff, cols - o0,
                (ldo & 7) == 0 && (ldp & 7) == 0);
    return;
  }
  const long long th = blockIdx.x * 8ll + warp;
  if (th >= static_cast<long long>(T) * H) return;
  const long long t = th / H;
  const int h = static_cast<int>(th - t * H);
  const A* pg = proj + t * ldp + g_off + h * V;
  A* o = out + t * ldo + h * V;
  if (h == H - 1)
    for (int i = H * V + lane; i < o0; i += 32) st_act(out + t * ldo + i, 0.f);
  const int req = tok_req[t];
  if (req < 0 || positions[t] < 0) {
    for (int c = lane; c < V; c += 32) st_act(o + c, 0.f);
    return;
  }
  const float m = mt[th];
  const float inv = 1.f / (fmaxf(fabsf(den[th]), expf(-m)) + 1e-6f);
  const float* x = num + th * V;
  const float* wh = w + h * V;
  float ss = 0.f;
  if ((V & 3) == 0 && (ldo & 3) == 0 && (ldp & 3) == 0) {
    for (int c = lane * 4; c < V; c += 128) {
      const float4 v = *reinterpret_cast<const float4*>(x + c);
      const float a0 = v.x * inv, a1 = v.y * inv, a2 = v.z * inv, a3 = v.w * inv;
      ss = fmaf(a0, a0, fmaf(a1, a1, fmaf(a2, a2, fmaf(a3, a3, ss))));
    }
    const float r = inv / sqrtf(warp_sum(ss) / static_cast<float>(V) + eps);
    for (int c = lane * 4; c < V; c += 128) {
      const float4 v = *reinterpret_cast<const float4*>(x + c), wv = *reinterpret_cast<const float4*>(wh + c);
      float y[4] = {v.x * r * wv.x, v.y * r * wv.y, v.z * r * wv.z, v.w * r * wv.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) y[i] /= 1.f + expf(-ld_act(pg + c + i));
      if (sizeof(A) == 2) {
        uint2 pk;
        *reinterpret_cast<__nv_bfloat162*>(&pk.x) = __floats2bfloat162_rn(y[0], y[1]);
        *reinterpret_cast<__nv_bfloat162*>(&pk.y) = __floats2bfloat162_rn(y[2], y[3]);
        *reinterpret_cast<uint2*>(o + c) = pk;
      } else {
        *reinterpret_cast<float4*>(o + c) = make_float4(y[0], y[1], y[2], y[3]);
      }
    }
  } else {
    for (int c = lane; c < V; c += 32) {
      const float v = x[c] * inv;
      ss = fmaf(v, v, ss);
    }
    const float r = inv / sqrtf(warp_sum(ss) / static_cast<float>(V) + eps);
    for (int c = lane; c < V; c += 32) st_act(o + c, x[c] * r * wh[c] / (1.f + expf(-ld_act(pg + c))));
  }
  if (positions[t] == last_pos[t] && lane == 0) m_state[static_cast<long long>(req) * H + h] = m;
}

}  // namespace stk

using namespace stk;

static MlstmArgs mlstm_args(const void* proj, long long ldp, int q_off, int k_off, int v_off, const float* gates,
                            const float* gate_bias, float cap, const int* query_start, const int* req_rows, const int* start_pos,
                            int n_req, float* S, float* n, float* m, float* num, float* den, float* mt, int heads, int dim,
                            int vdim) {
  MlstmArgs a;
  a.proj = proj; a.ldp = ldp; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off;
  a.gates = gates; a.gate_bias = gate_bias; a.cap = cap;
  a.query_start = query_start; a.req_rows = req_rows; a.start_pos = start_pos; a.n_req = n_req;
  a.S = S; a.n = n; a.m = m;
  a.num = num; a.den = den; a.mt = mt;
  a.H = heads; a.D = dim; a.V = vdim;
  return a;
}

// Spans of min_span .. max_span tokens, token by token.
STK_API int stk_mlstm_scan(const void* proj, long long ldp, int q_off, int k_off, int v_off, const float* gates,
                           const float* gate_bias, float cap, const int* query_start, const int* req_rows, const int* start_pos,
                           int n_req, float* S, float* n, float* m, float* num, float* den, float* mt, int heads, int dim,
                           int vdim, int fp32, int min_span, int max_span, int T, void* stream) {
  if (T <= 0 || n_req <= 0) return 0;
  if (heads < 1 || dim < 1 || dim > 1024 || vdim < 1 || heads > 65535 || n_req > 65535) return -1;
  const MlstmArgs a = mlstm_args(proj, ldp, q_off, k_off, v_off, gates, gate_bias, cap, query_start, req_rows, start_pos, n_req, S,
                                 n, m, num, den, mt, heads, dim, vdim);
  const size_t smem = (static_cast<size_t>(dim) * (kScanCols + 3) + 8 * kScanCols) * sizeof(float);
  if (cudaFuncSetAttribute(mlstm_scan_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) != cudaSuccess ||
      cudaFuncSetAttribute(mlstm_scan_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) !=
          cudaSuccess)
    return -3;
  const dim3 grid((vdim + kScanCols - 1) / kScanCols, heads, n_req);
  cudaStream_t st = (cudaStream_t)stream;
  if (fp32) launch_pdl(mlstm_scan_kernel<float>, grid, dim3(256), smem, st, a, min_span, max_span);
  else launch_pdl(mlstm_scan_kernel<__nv_bfloat16>, grid, dim3(256), smem, st, a, min_span, max_span);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_mlstm_gate_slot() { return kGateSlot; }
STK_API long long stk_mlstm_state_slot(int dim, int vdim) { return state_slot_floats(dim, vdim); }

// Spans of at least min_span tokens in chunks of 64 (bf16).  max_chunks bounds their number over all requests;
// fp32 work space: gate_ws [max_chunks * heads * stk_mlstm_gate_slot()], states [max_chunks * heads * stk_mlstm_state_slot()].
STK_API int stk_mlstm_chunks(const void* proj, long long ldp, int q_off, int k_off, int v_off, const float* gates,
                             const float* gate_bias, float cap, const int* query_start, const int* req_rows, const int* start_pos,
                             int n_req, float* S, float* n, float* m, float* num, float* den, float* mt, int heads, int dim,
                             int vdim, int min_span, float* gate_ws, float* states, int max_chunks, int T, void* stream) {
  if (T <= 0 || n_req <= 0 || max_chunks <= 0) return 0;
  if (heads < 1 || dim < 1 || dim > 256 || vdim < 1 || heads > 65535 || static_cast<long long>(heads) * n_req > 65535 ||
      max_chunks > 65535 || min_span < 1 || (reinterpret_cast<uintptr_t>(states) & 15))
    return -1;
  const MlstmArgs a = mlstm_args(proj, ldp, q_off, k_off, v_off, gates, gate_bias, cap, query_start, req_rows, start_pos, n_req, S,
                                 n, m, num, den, mt, heads, dim, vdim);
  const int ks = (dim + 15) / 16 * 16 + 8;
  const size_t smem2 = static_cast<size_t>(6) * kChunk * kStStride * 2;
  const size_t tail = static_cast<size_t>(kChunk) * ks > 4u * kOutRows * kOutStride ? static_cast<size_t>(kChunk) * ks
                                                                                 : 4u * kOutRows * kOutStride;
  const size_t smem3 = (static_cast<size_t>(kChunk) * (ks + kOutStride + 2 * kStStride) + tail) * 2;
  if (cudaFuncSetAttribute(mlstm_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024) != cudaSuccess ||
      cudaFuncSetAttribute(mlstm_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024) != cudaSuccess)
    return -3;
  cudaStream_t st = (cudaStream_t)stream;
  launch_pdl(mlstm_chunk_gates_kernel, dim3(heads, n_req), dim3(256), 0, st, a, min_span, gate_ws);
  launch_pdl(mlstm_chunk_state_kernel, dim3((vdim + 63) / 64, (dim + 63) / 64, heads * n_req), dim3(128), smem2, st, a, min_span,
             gate_ws, states);
  launch_pdl(mlstm_chunk_out_kernel, dim3((vdim + kOutCols - 1) / kOutCols, max_chunks, heads), dim3(256), smem3, st, a, min_span,
             gate_ws, states);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_mlstm_finish(const float* num, const float* den, const float* mt, float* m_state, const float* norm_w, float eps,
                             const int* tok_req, const int64_t* positions, const int* last_pos, const void* proj, long long ldp,
                             int g_off, void* out, long long ldo, int fp32, int heads, int vdim, int gate_off, int up_off, int ff,
                             int ff_off, int cols, int T, void* stream) {
  if (T <= 0) return 0;
  const int n = cols - ff_off;
  const int head_blocks = static_cast<int>((static_cast<long long>(T) * heads + 7) / 8), ff_blocks = n > 0 ? (n + 2047) / 2048 : 0;
  const dim3 grid(head_blocks + T * ff_blocks);
  cudaStream_t st = (cudaStream_t)stream;
  if (fp32)
    launch_pdl(mlstm_finish_kernel<float>, grid, dim3(256), 0, st, num, den, mt, m_state, norm_w, eps, tok_req, positions,
               last_pos, (const float*)proj, ldp, g_off, (float*)out, ldo, heads, vdim, gate_off, up_off, ff, ff_off, cols, T,
               head_blocks, ff_blocks);
  else
    launch_pdl(mlstm_finish_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, num, den, mt, m_state, norm_w, eps, tok_req, positions,
               last_pos, (const __nv_bfloat16*)proj, ldp, g_off, (__nv_bfloat16*)out, ldo, heads, vdim, gate_off, up_off, ff,
               ff_off, cols, T, head_blocks, ff_blocks);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
