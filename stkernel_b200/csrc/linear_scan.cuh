// Linear recurrences with a scalar decay per head and token,
//
//   S_t = exp(g_t) S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t  (+ skip v_t)        S [D, V] fp32 per head and request row
//
// shared by retention (retention.cu) and Mamba-2 (mamba2.cu), and with a decay per key channel and a bonus for the current token, read out
// before the update, by time mixing (time_mix.cu).  A span that starts at position 0 starts from a zero state.
//
//   linear_scan_kernel     token by token, any size and type: one CTA per (32 or 64 value columns, head, request), the block of the
//                          state in registers.  A `Front` supplies a token's q and k (in shared memory), v and decay, so that
//                          rotations and input weights happen on the way in.
//   linear_chunk_*         spans of some length, bf16 operands (linear_scan.cu)
#pragma once
#include "hybrid_block.cuh"

namespace stk {

struct ScanArgs {
  const int* query_start; const int* req_rows; const int* start_pos; int n_req;
  float* S; float* o;                             // state [rows, H, D, V]; outputs [T, H, V]
  int H, D, V;
};

constexpr int kScanThreads = 256, kScanRows = 8;

// ---- chunked form: the states before every chunk (linear_scan.cu) --------------------------------
// A state is kept in the layout of the B operand of the output products: per block of 16 value rows x 16 state rows 32 lanes x 16 bytes of
// high parts, then of remainders.
__host__ __device__ inline int blocks16(int n) { return (n + 15) / 16; }
constexpr int kBlockFloats = 256;                // a 16 x 16 block as a bf16 pair
__host__ __device__ inline long long linear_slot_floats(int D, int V) {
  return static_cast<long long>(blocks16(D)) * blocks16(V) * kBlockFloats;
}
// States of a recurrence whose state rows decay by factors of their own (channel [chunk][H][D]) from chunk to chunk: S_end = diag(f) S +
// sum_j k_j v_j^T with keys (high parts kh, remainders kl) that already carry the decay from their token to the end of the chunk.
int linear_states_per_channel(const __nv_bfloat16* kh, const __nv_bfloat16* kl, long long ldk, int step, int width, const __nv_bfloat16* v,
                              long long ldv, int v_off, const float* channel, const ScanArgs& s, int min_span, float* states, int T,
                              cudaStream_t st);

// Front:
//   float2 fill(t, pos, h, q, k)   token t at position pos, all threads; returns the decay and what its rounding left over (the same
//                                  small error at every token would add up over many)
//   or, kPerChannel: void fill(t, h, q, k, uk, w) with the bonus' keys and the channels' decays as well
//   float value(t, h, col)         v
//   float skip(h)                  factor of v in the output
template <typename Front, int NR, int VEC>
__global__ void __launch_bounds__(kScanThreads)
linear_scan_kernel(const Front f, const ScanArgs a, int min_span, int max_span) {
  extern __shared__ __align__(16) float sm[];
  constexpr int kCols = 32 * VEC;
  float* q = sm;                                  // [D]
  float* k = q + a.D;                             // [D]
  float* x = k + a.D;                             // [kCols] v
  float* part = x + kCols;                        // [8][kCols]
  float* uk = part + kScanRows * kCols;           // per channel: [D] bonus' keys, [D] decays
  float2* w = reinterpret_cast<float2*>(uk + (a.D + 1) / 2 * 2);
  pdl_wait();
  pdl_trigger();
  const int vb = blockIdx.x, h = blockIdx.y, ri = blockIdx.z;
  const int q0 = a.query_start[ri], span = a.query_start[ri + 1] - q0;
  if (span <= 0 || span < min_span || span > max_span) return;
  const long long row = a.req_rows[ri];
  const int start = a.start_pos[ri];
  const int lane = threadIdx.x & 31, r = threadIdx.x >> 5;
  const int col = vb * kCols + lane * VEC;
  float* gS = a.S + (row * a.H + h) * static_cast<long long>(a.D) * a.V + col;
  float S[NR][VEC];
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = r + j * kScanRows;
    const bool in = start != 0 && d < a.D;
    if (VEC == 2 && in && col + 1 < a.V) {
      const float2 s = *reinterpret_cast<const float2*>(gS + static_cast<long long>(d) * a.V);
      S[j][0] = s.x;
      S[j][VEC - 1] = s.y;
    } else {
#pragma unroll
      for (int c = 0; c < VEC; ++c) S[j][c] = in && col + c < a.V ? gS[static_cast<long long>(d) * a.V + c] : 0.f;
    }
  }
  const float skip = f.skip(h);
  for (int i = 0; i < span; ++i) {
    const long long t = q0 + i;
    __syncthreads();
    float2 decay = make_float2(0.f, 0.f);
    if constexpr (Front::kPerChannel) f.fill(t, h, q, k, uk, w);
    else decay = f.fill(t, start + i, h, q, k);
    float v[VEC];
#pragma unroll
    for (int c = 0; c < VEC; ++c) {
      v[c] = col + c < a.V ? f.value(t, h, col + c) : 0.f;
      if (r == 0) x[lane * VEC + c] = v[c];
    }
    __syncthreads();
    float acc[VEC];
#pragma unroll
    for (int c = 0; c < VEC; ++c) acc[c] = 0.f;
#pragma unroll
    for (int j = 0; j < NR; ++j) {
      const int d = r + j * kScanRows;
      if (d < a.D) {
        const float kd = k[d], qd = q[d];
        if constexpr (Front::kPerChannel) {
          const float ud = uk[d];
          const float2 wd = w[d];
#pragma unroll
          for (int c = 0; c < VEC; ++c) {
            acc[c] = fmaf(qd, fmaf(ud, v[c], S[j][c]), acc[c]);
            S[j][c] = fmaf(wd.x, S[j][c], fmaf(wd.y, S[j][c], kd * v[c]));
          }
        } else {
#pragma unroll
          for (int c = 0; c < VEC; ++c) {
            S[j][c] = fmaf(decay.x, S[j][c], fmaf(decay.y, S[j][c], kd * v[c]));
            acc[c] = fmaf(qd, S[j][c], acc[c]);
          }
        }
      }
    }
#pragma unroll
    for (int c = 0; c < VEC; ++c) part[r * kCols + lane * VEC + c] = acc[c];
    __syncthreads();
    const int oc = threadIdx.x;
    if (oc < kCols && vb * kCols + oc < a.V) {
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < kScanRows; ++w) s += part[w * kCols + oc];
      a.o[(t * a.H + h) * a.V + vb * kCols + oc] = fmaf(skip, x[oc], s);
    }
  }
#pragma unroll
  for (int j = 0; j < NR; ++j) {
    const int d = r + j * kScanRows;
    if (d >= a.D) continue;
    if (VEC == 2 && col + 1 < a.V) {
      *reinterpret_cast<float2*>(gS + static_cast<long long>(d) * a.V) = make_float2(S[j][0], S[j][VEC - 1]);
    } else {
#pragma unroll
      for (int c = 0; c < VEC; ++c)
        if (col + c < a.V) gS[static_cast<long long>(d) * a.V + c] = S[j][c];
    }
  }
}

template <typename Front, int NR, int VEC>
static int launch_scan_as(const Front& f, const ScanArgs& a, int min_span, int max_span, cudaStream_t st) {
  constexpr int kCols = 32 * VEC;
  // kCols is even: everything behind q, k starts on 8 bytes when D is rounded up to even
  const size_t smem = static_cast<size_t>(2 * a.D + (1 + kScanRows) * kCols + (Front::kPerChannel ? 3 * a.D + 2 : 0)) * sizeof(float);
  launch_pdl(linear_scan_kernel<Front, NR, VEC>, dim3((a.V + kCols - 1) / kCols, a.H, a.n_req), dim3(kScanThreads), smem, st, f, a,
             min_span, max_span);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// Spans of min_span .. max_span tokens, D up to 1024.
template <typename Front>
static int launch_scan(const Front& f, const ScanArgs& a, int min_span, int max_span, cudaStream_t st) {
  if (a.H < 1 || a.H > 65535 || a.D < 1 || a.D > 1024 || a.V < 1 || a.n_req > 65535) return -1;
  if (a.n_req <= 0) return 0;
  const bool two = a.V >= 64 && a.V % 2 == 0;
  if (a.D <= 64) return two ? launch_scan_as<Front, 8, 2>(f, a, min_span, max_span, st) : launch_scan_as<Front, 8, 1>(f, a, min_span, max_span, st);
  if (a.D <= 128) return two ? launch_scan_as<Front, 16, 2>(f, a, min_span, max_span, st) : launch_scan_as<Front, 16, 1>(f, a, min_span, max_span, st);
  if (a.D <= 256) return launch_scan_as<Front, 32, 1>(f, a, min_span, max_span, st);
  return launch_scan_as<Front, 128, 1>(f, a, min_span, max_span, st);
}

}  // namespace stk
