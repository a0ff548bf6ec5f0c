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
//                       (1) per chunk: sum_j exp(a_j - A) k_j v_j^T, A = max_j a_j;  (2) a scan over the chunks turns these into
//                       the state before each chunk;  (3) per chunk: the outputs.  (1) and (3) run on the tensor cores with the
//                       fp32 operand of each product as a bf16 pair (16 mantissa bits).
// Sums of log gates reach hundreds, so they are formed in fp64 and kept as integer part + remainder: differences lose nothing.
#define STK_PDL_CLASS 16
#include "common.cuh"

namespace stk {

constexpr int kChunk = 64;
constexpr int kGateSlot = 3 * kChunk + 8;      // a (integer, remainder), F, then A, F_end, m_start as (integer, remainder) pairs

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
__device__ __forceinline__ void ml_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void ml_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

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
__device__ __forceinline__ void mls_ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mls_ldsm4_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mls_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mls_split(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16(x);
  lo = __float2bfloat16(x - bf16_to_f(hi));
}
__device__ __forceinline__ void mls_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 r = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&r);
}

// chunk index of the step -> (request, first chunk of the request, tokens [t0, t0 + n) of the step); false past the end
struct ChunkRef { int ri, first, t0, n; };
__device__ __forceinline__ bool find_chunk(const MlstmArgs& a, int min_span, int ci, ChunkRef& c) {
  int base = 0;
  for (int i = 0; i < a.n_req; ++i) {
    const int q0 = a.query_start[i], span = a.query_start[i + 1] - q0;
    if (span < min_span) continue;
    const int nc = (span + kChunk - 1) / kChunk;
    if (ci < base + nc) {
      c.ri = i;
      c.first = base;
      c.t0 = q0 + (ci - base) * kChunk;
      c.n = min(kChunk, span - (ci - base) * kChunk);
      return true;
    }
    base += nc;
  }
  return false;
}

// rows [0, 64) x cols [0, width) of head columns into shared memory; rows >= n and columns >= width up to `cols` are zero
__device__ __forceinline__ void load_rows(__nv_bfloat16* dst, int stride, int cols, const __nv_bfloat16* src, long long ld, int n,
                                          int width, int nthreads) {
  if ((width & 7) == 0 && (cols & 7) == 0 && (ld & 7) == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0) {
    const int ch = cols >> 3;
    for (int e = threadIdx.x; e < kChunk * ch; e += nthreads) {
      const int r = e / ch, c = (e - r * ch) * 8;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < n && c < width) v = *reinterpret_cast<const uint4*>(src + r * ld + c);
      *reinterpret_cast<uint4*>(dst + r * stride + c) = v;
    }
  } else {
    for (int e = threadIdx.x; e < kChunk * cols; e += nthreads) {
      const int r = e / cols, c = e - r * cols;
      dst[r * stride + c] = r < n && c < width ? src[r * ld + c] : __float2bfloat16(0.f);
    }
  }
}

// (1) per chunk and 64 value columns: U = sum_j exp(a_j - A) k_j v_j^T, and (first column block) u = sum_j exp(a_j - A) k_j and
// the chunk's gate record.  states: [chunk][H][D * V + D].
__global__ void __launch_bounds__(128)
mlstm_chunk_state_kernel(const MlstmArgs a, int min_span, float* __restrict__ gate_ws, float* __restrict__ states) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ float s_w[kChunk];
  __shared__ double s_f[kChunk], s_i[kChunk];
  __shared__ ChunkRef s_c;
  __shared__ int s_ok;
  const int Dp = (a.D + 15) / 16 * 16, ks = Dp + 8, vs = 72;
  __nv_bfloat16* k = reinterpret_cast<__nv_bfloat16*>(smem_raw);        // [64][Dp + 8]
  __nv_bfloat16* vh = k + kChunk * ks;                                  // [64][72] weighted values, high part
  __nv_bfloat16* vl = vh + kChunk * vs;                                 // remainder
  pdl_wait();
  pdl_trigger();
  const int vb = blockIdx.x, ci = blockIdx.y, h = blockIdx.z;
  if (threadIdx.x == 0) s_ok = find_chunk(a, min_span, ci, s_c) ? 1 : 0;
  __syncthreads();
  if (!s_ok) return;
  const ChunkRef c = s_c;
  const __nv_bfloat16* p = reinterpret_cast<const __nv_bfloat16*>(a.proj) + c.t0 * a.ldp;
  if (threadIdx.x < kChunk) {
    float ig = 0.f, fg = 0.f;
    if (threadIdx.x < c.n) log_gates(a, c.t0 + threadIdx.x, h, ig, fg);
    s_i[threadIdx.x] = ig;
    s_f[threadIdx.x] = fg;
  }
  load_rows(k, ks, Dp, p + a.k_off + h * a.D, a.ldp, c.n, a.D, 128);
  __syncthreads();
  if (threadIdx.x < 32) {
    // running sum of the log forget gates over 64 tokens, two per lane
    const int l = threadIdx.x;
    const double f0 = s_f[2 * l], f1 = f0 + s_f[2 * l + 1];
    double inc = f1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double up = __shfl_up_sync(0xffffffffu, inc, o);
      if (l >= o) inc += up;
    }
    const double before = inc - f1;
    s_f[2 * l] = before + f0;
    s_f[2 * l + 1] = inc;
    const double a0 = 2 * l < c.n ? s_i[2 * l] - s_f[2 * l] : -1e300, a1 = 2 * l + 1 < c.n ? s_i[2 * l + 1] - s_f[2 * l + 1] : -1e300;
    double mx = a0 > a1 ? a0 : a1;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const double other = __shfl_xor_sync(0xffffffffu, mx, o);
      mx = other > mx ? other : mx;
    }
    s_w[2 * l] = 2 * l < c.n ? expf(static_cast<float>(a0 - mx)) : 0.f;
    s_w[2 * l + 1] = 2 * l + 1 < c.n ? expf(static_cast<float>(a1 - mx)) : 0.f;
    if (vb == 0) {
      float* g = gate_ws + (static_cast<long long>(ci) * a.H + h) * kGateSlot;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int j = 2 * l + i;
        const double av = i == 0 ? a0 : a1;
        const double ai = j < c.n ? rint(av) : -1e30;
        g[j] = static_cast<float>(ai);
        g[kChunk + j] = j < c.n ? static_cast<float>(av - ai) : 0.f;
        g[2 * kChunk + j] = static_cast<float>(s_f[j]);
      }
      if (l == 0) {
        const double ai = rint(mx);
        g[3 * kChunk + 0] = static_cast<float>(ai);
        g[3 * kChunk + 1] = static_cast<float>(mx - ai);
      }
      __syncwarp();
      if (l == 0) {
        const double fe = s_f[c.n - 1], fi = rint(fe);
        g[3 * kChunk + 2] = static_cast<float>(fi);
        g[3 * kChunk + 3] = static_cast<float>(fe - fi);
      }
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < kChunk * 64; e += 128) {
    const int r = e >> 6, cc = e & 63, col = vb * 64 + cc;
    const float v = r < c.n && col < a.V ? bf16_to_f(p[r * a.ldp + a.v_off + h * a.V + col]) * s_w[r] : 0.f;
    mls_split(v, vh[r * vs + cc], vl[r * vs + cc]);
  }
  __syncthreads();
  float* U = states + (static_cast<long long>(ci) * a.H + h) * (static_cast<long long>(a.D) * a.V + a.D);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int mt = warp; mt < Dp / 16; mt += 4) {
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[j][i] = 0.f;
#pragma unroll
    for (int kk = 0; kk < kChunk / 16; ++kk) {
      uint32_t af[4];
      mls_ldsm4_t(af, k + (kk * 16 + (lane & 7) + (lane >> 4) * 8) * ks + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        uint32_t bh[4], bl[4];
        const int off = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + j * 16 + (lane >> 4) * 8;
        mls_ldsm4_t(bh, vh + off);
        mls_ldsm4_t(bl, vl + off);
        mls_mma(acc[2 * j], af, bh[0], bh[1]);
        mls_mma(acc[2 * j + 1], af, bh[2], bh[3]);
        mls_mma(acc[2 * j], af, bl[0], bl[1]);
        mls_mma(acc[2 * j + 1], af, bl[2], bl[3]);
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = mt * 16 + (lane >> 2) + (i >> 1) * 8, col = vb * 64 + j * 8 + (lane & 3) * 2 + (i & 1);
        if (d < a.D && col < a.V) U[static_cast<long long>(d) * a.V + col] = acc[j][i];
      }
  }
  if (vb == 0) {
    float* un = U + static_cast<long long>(a.D) * a.V;
    for (int d = threadIdx.x; d < a.D; d += 128) {
      float s = 0.f;
      for (int j = 0; j < c.n; ++j) s = fmaf(s_w[j], bf16_to_f(k[j * ks + d]), s);
      un[d] = s;
    }
  }
}

// (2) scan over the chunks of each request: states[c] becomes the state before chunk c, the request's stored state advances.
__global__ void __launch_bounds__(256)
mlstm_chunk_scan_kernel(const MlstmArgs a, int min_span, float* __restrict__ gate_ws, float* __restrict__ states) {
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.y, ri = blockIdx.z;
  const int span = a.query_start[ri + 1] - a.query_start[ri];
  if (span < min_span || span <= 0) return;
  int first = 0;
  for (int i = 0; i < ri; ++i) {
    const int s = a.query_start[i + 1] - a.query_start[i];
    if (s >= min_span) first += (s + kChunk - 1) / kChunk;
  }
  const int nc = (span + kChunk - 1) / kChunk;
  const long long row = a.req_rows[ri];
  const bool fresh = a.start_pos[ri] == 0;
  const long long dv = static_cast<long long>(a.D) * a.V, total = dv + a.D;
  const long long e = blockIdx.x * 256ll + threadIdx.x;
  const bool ok = e < total;
  float* dst = e < dv ? a.S + (row * a.H + h) * dv + e : a.n + (row * a.H + h) * a.D + (e - dv);
  float s = ok && !fresh ? *dst : 0.f;
  double m = fresh ? 0.0 : static_cast<double>(a.m[row * a.H + h]);
  for (int c = 0; c < nc; ++c) {
    const long long slot = static_cast<long long>(first + c) * a.H + h;
    float* g = gate_ws + slot * kGateSlot + 3 * kChunk;
    const double A = static_cast<double>(g[0]) + g[1], F = static_cast<double>(g[2]) + g[3];
    if (e == 0) {
      const double mi = rint(m);
      g[4] = static_cast<float>(mi);
      g[5] = static_cast<float>(m - mi);
    }
    const double M = m > A ? m : A;
    const float fs = expf(static_cast<float>(m - M)), fu = expf(static_cast<float>(A - M));
    if (ok) {
      float* u = states + slot * total + e;
      const float x = *u;
      *u = s;
      s = fmaf(fs, s, fu * x);
    }
    m = F + M;
  }
  if (ok) *dst = s;
}

// (3) outputs of a chunk for 64 value columns; the first column block also writes n_t . q_t and m_t.
__global__ void __launch_bounds__(128)
mlstm_chunk_out_kernel(const MlstmArgs a, int min_span, const float* __restrict__ gate_ws, const float* __restrict__ states) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  __shared__ float s_ai[kChunk], s_ar[kChunk], s_mi[kChunk], s_mr[kChunk], s_in[kChunk], s_nq[kChunk];
  __shared__ ChunkRef s_c;
  __shared__ int s_ok;
  const int Dp = (a.D + 15) / 16 * 16, ks = Dp + 8, vs = 72;
  __nv_bfloat16* q = reinterpret_cast<__nv_bfloat16*>(smem_raw);        // [64][Dp + 8]
  __nv_bfloat16* k = q + kChunk * ks;
  __nv_bfloat16* v = k + kChunk * ks;                                   // [64][72]
  __nv_bfloat16* sh = v + kChunk * vs;                                  // 64 rows of the state, high part
  __nv_bfloat16* sl = sh + 64 * vs;                                     // remainder
  pdl_wait();
  pdl_trigger();
  const int vb = blockIdx.x, ci = blockIdx.y, h = blockIdx.z;
  if (threadIdx.x == 0) s_ok = find_chunk(a, min_span, ci, s_c) ? 1 : 0;
  __syncthreads();
  if (!s_ok) return;
  const ChunkRef c = s_c;
  const __nv_bfloat16* p = reinterpret_cast<const __nv_bfloat16*>(a.proj) + c.t0 * a.ldp;
  const long long slot = static_cast<long long>(ci) * a.H + h;
  const float* g = gate_ws + slot * kGateSlot;
  const long long dv = static_cast<long long>(a.D) * a.V;
  const float* S0 = states + slot * (dv + a.D);
  load_rows(q, ks, Dp, p + a.q_off + h * a.D, a.ldp, c.n, a.D, 128);
  load_rows(k, ks, Dp, p + a.k_off + h * a.D, a.ldp, c.n, a.D, 128);
  load_rows(v, vs, 64, p + a.v_off + h * a.V + vb * 64, a.ldp, c.n, min(64, a.V - vb * 64), 128);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0) {
    // M_t = max(m_start, running max of a): pairs compared through their sum in fp64, two tokens per lane
    const double m0 = static_cast<double>(g[3 * kChunk + 4]) + g[3 * kChunk + 5];
    const double a0 = static_cast<double>(g[2 * lane]) + g[kChunk + 2 * lane];
    const double a1 = static_cast<double>(g[2 * lane + 1]) + g[kChunk + 2 * lane + 1];
    const double pm = a0 > a1 ? a0 : a1;
    double inc = pm;
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
  __syncthreads();
  const float qs = 1.f / sqrtf(static_cast<float>(a.D));
  if (vb == 0) {
    const float* n0 = S0 + dv;
    for (int r = warp * 16; r < warp * 16 + 16; ++r) {
      float s = 0.f;
      for (int d = lane; d < a.D; d += 32) s = fmaf(bf16_to_f(q[r * ks + d]), n0[d], s);
      s = warp_sum(s);
      if (lane == 0) s_nq[r] = s;
    }
    __syncwarp();
  }
  // inter-chunk part: q S_start, 64 state rows at a time
  float o[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[j][i] = 0.f;
  for (int d0 = 0; d0 < Dp; d0 += 64) {
    __syncthreads();
    for (int e = threadIdx.x; e < 64 * 64; e += 128) {
      const int d = d0 + (e >> 6), col = vb * 64 + (e & 63);
      const float x = d < a.D && col < a.V ? S0[static_cast<long long>(d) * a.V + col] : 0.f;
      mls_split(x, sh[(e >> 6) * vs + (e & 63)], sl[(e >> 6) * vs + (e & 63)]);
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      if (d0 + kk * 16 < Dp) {
        uint32_t af[4];
        mls_ldsm4(af, q + (warp * 16 + (lane & 15)) * ks + d0 + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          uint32_t bh[4], bl[4];
          const int off = (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + j * 16 + (lane >> 4) * 8;
          mls_ldsm4_t(bh, sh + off);
          mls_ldsm4_t(bl, sl + off);
          mls_mma(o[2 * j], af, bh[0], bh[1]);
          mls_mma(o[2 * j + 1], af, bh[2], bh[3]);
          mls_mma(o[2 * j], af, bl[0], bl[1]);
          mls_mma(o[2 * j + 1], af, bl[2], bl[3]);
        }
      }
    }
  }
  int row[2];
  float mi[2], mr[2], sum[2] = {0.f, 0.f};
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    row[r] = warp * 16 + (lane >> 2) + r * 8;
    mi[r] = s_mi[row[r]];
    mr[r] = s_mr[row[r]];
  }
#pragma unroll
  for (int j = 0; j < 8; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) o[j][i] *= s_in[row[i >> 1]];
  // intra-chunk part, 16 keys at a time up to the warp's own tokens
  for (int kb = 0; kb <= warp; ++kb) {
    float s[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) s[j][i] = 0.f;
    for (int kk = 0; kk < Dp / 16; ++kk) {
      uint32_t af[4], bf[4];
      mls_ldsm4(af, q + (warp * 16 + (lane & 15)) * ks + kk * 16 + (lane >> 4) * 8);
      mls_ldsm4(bf, k + (kb * 16 + (lane >> 4) * 8 + (lane & 7)) * ks + kk * 16 + ((lane >> 3) & 1) * 8);
      mls_mma(s[0], af, bf[0], bf[1]);
      mls_mma(s[1], af, bf[2], bf[3]);
    }
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int col = kb * 16 + j * 8 + (lane & 3) * 2 + (i & 1), r = i >> 1;
        const float w = col <= row[r] ? expf((s_ai[col] - mi[r]) + (s_ar[col] - mr[r])) : 0.f;
        s[j][i] *= w;
        sum[r] += s[j][i];
      }
    uint32_t hi[4], lo[4];
    mls_split2(s[0][0], s[0][1], hi[0], lo[0]);
    mls_split2(s[0][2], s[0][3], hi[1], lo[1]);
    mls_split2(s[1][0], s[1][1], hi[2], lo[2]);
    mls_split2(s[1][2], s[1][3], hi[3], lo[3]);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      uint32_t bf[4];
      mls_ldsm4_t(bf, v + (kb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * vs + j * 16 + (lane >> 4) * 8);
      mls_mma(o[2 * j], hi, bf[0], bf[1]);
      mls_mma(o[2 * j + 1], hi, bf[2], bf[3]);
      mls_mma(o[2 * j], lo, bf[0], bf[1]);
      mls_mma(o[2 * j + 1], lo, bf[2], bf[3]);
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
    sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
    if (row[r] >= c.n) continue;
    const long long t = c.t0 + row[r];
    if (vb == 0 && (lane & 3) == 0) a.den[t * a.H + h] = (sum[r] + s_in[row[r]] * s_nq[row[r]]) * qs;
    float* out = a.num + (t * a.H + h) * a.V + vb * 64;
#pragma unroll
    for (int j = 0; j < 8; ++j)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int cc = j * 8 + (lane & 3) * 2 + i;
        if (vb * 64 + cc < a.V) out[cc] = o[j][2 * r + i] * qs;
      }
  }
}

// ---- head norm, output gate, stored maximum, feed-forward activation -----------------------------------
// blockIdx.x == 0: out[t, h * V + c] = o / rms(o over the head) * w * sigmoid(g), o = num / (max(|den|, exp(-m)) + 1e-6).
// blockIdx.x > 0: 2048 columns each of the feed-forward half (silu(gate) * up, zero padding), as join_glu.
template <typename A>
__global__ void __launch_bounds__(256)
mlstm_finish_kernel(const float* __restrict__ num, const float* __restrict__ den, const float* __restrict__ mt,
                    float* __restrict__ m_state, const float* __restrict__ w, float eps, const int* __restrict__ tok_req,
                    const int64_t* __restrict__ positions, const int* __restrict__ last_pos, const A* __restrict__ proj,
                    long long ldp, int g_off, A* __restrict__ out, long long ldo, int H, int V, int go, int uo, int ff, int o0,
                    int cols) {
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.y;
  const A* p = proj + t * ldp;
  A* o = out + t * ldo;
  if (blockIdx.x > 0) {
    const int n = cols - o0;
    for (int j = (blockIdx.x - 1) * 2048 + threadIdx.x; j < min(n, static_cast<int>(blockIdx.x) * 2048); j += 256) {
      float v = 0.f;
      if (j < ff) {
        const float g = ml_f(p[go + j]);
        v = g / (1.f + expf(-g)) * ml_f(p[uo + j]);
      }
      ml_st(o + o0 + j, v);
    }
    return;
  }
  for (int i = H * V + threadIdx.x; i < o0; i += 256) ml_st(o + i, 0.f);
  const int req = tok_req[t];
  const bool ok = req >= 0 && positions[t] >= 0;
  const bool last = ok && positions[t] == last_pos[t];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int h = warp; h < H; h += 8) {
    if (!ok) {
      for (int c = lane; c < V; c += 32) ml_st(o + h * V + c, 0.f);
      continue;
    }
    const float m = mt[t * H + h];
    const float inv = 1.f / (fmaxf(fabsf(den[t * H + h]), expf(-m)) + 1e-6f);
    const float* x = num + (t * H + h) * V;
    float ss = 0.f;
    for (int c = lane; c < V; c += 32) {
      const float v = x[c] * inv;
      ss = fmaf(v, v, ss);
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(V) + eps);
    for (int c = lane; c < V; c += 32) {
      const float g = ml_f(p[g_off + h * V + c]);
      ml_st(o + h * V + c, x[c] * inv * r * w[h * V + c] / (1.f + expf(-g)));
    }
    if (last && lane == 0) m_state[static_cast<long long>(req) * H + h] = m;
  }
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

// Spans of at least min_span tokens in chunks of 64 (bf16).  max_chunks bounds their number over all requests;
// gate_ws [max_chunks * heads * stk_mlstm_gate_slot()], states [max_chunks * heads * (dim * vdim + dim)].
STK_API int stk_mlstm_chunks(const void* proj, long long ldp, int q_off, int k_off, int v_off, const float* gates,
                             const float* gate_bias, float cap, const int* query_start, const int* req_rows, const int* start_pos,
                             int n_req, float* S, float* n, float* m, float* num, float* den, float* mt, int heads, int dim,
                             int vdim, int min_span, float* gate_ws, float* states, int max_chunks, int T, void* stream) {
  if (T <= 0 || n_req <= 0 || max_chunks <= 0) return 0;
  if (heads < 1 || dim < 1 || dim > 256 || vdim < 1 || heads > 65535 || n_req > 65535 || max_chunks > 65535 || min_span < 1)
    return -1;
  const MlstmArgs a = mlstm_args(proj, ldp, q_off, k_off, v_off, gates, gate_bias, cap, query_start, req_rows, start_pos, n_req, S,
                                 n, m, num, den, mt, heads, dim, vdim);
  const int Dp = (dim + 15) / 16 * 16;
  const size_t smem1 = static_cast<size_t>(kChunk) * (Dp + 8 + 2 * 72) * 2;
  const size_t smem3 = static_cast<size_t>(kChunk) * (2 * (Dp + 8) + 3 * 72) * 2;
  if (cudaFuncSetAttribute(mlstm_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024) != cudaSuccess ||
      cudaFuncSetAttribute(mlstm_chunk_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024) != cudaSuccess)
    return -3;
  const dim3 grid((vdim + 63) / 64, max_chunks, heads);
  const long long total = static_cast<long long>(dim) * vdim + dim;
  cudaStream_t st = (cudaStream_t)stream;
  launch_pdl(mlstm_chunk_state_kernel, grid, dim3(128), smem1, st, a, min_span, gate_ws, states);
  launch_pdl(mlstm_chunk_scan_kernel, dim3((total + 255) / 256, heads, n_req), dim3(256), 0, st, a, min_span, gate_ws, states);
  launch_pdl(mlstm_chunk_out_kernel, grid, dim3(128), smem3, st, a, min_span, gate_ws, states);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_mlstm_finish(const float* num, const float* den, const float* mt, float* m_state, const float* norm_w, float eps,
                             const int* tok_req, const int64_t* positions, const int* last_pos, const void* proj, long long ldp,
                             int g_off, void* out, long long ldo, int fp32, int heads, int vdim, int gate_off, int up_off, int ff,
                             int ff_off, int cols, int T, void* stream) {
  if (T <= 0) return 0;
  if (T > 65535) return -1;
  const int n = cols - ff_off;
  const dim3 grid(1 + (n > 0 ? (n + 2047) / 2048 : 0), T);
  cudaStream_t st = (cudaStream_t)stream;
  if (fp32)
    launch_pdl(mlstm_finish_kernel<float>, grid, dim3(256), 0, st, num, den, mt, m_state, norm_w, eps, tok_req, positions,
               last_pos, (const float*)proj, ldp, g_off, (float*)out, ldo, heads, vdim, gate_off, up_off, ff, ff_off, cols);
  else
    launch_pdl(mlstm_finish_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, num, den, mt, m_state, norm_w, eps, tok_req, positions,
               last_pos, (const __nv_bfloat16*)proj, ldp, g_off, (__nv_bfloat16*)out, ldo, heads, vdim, gate_off, up_off, ff,
               ff_off, cols);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
