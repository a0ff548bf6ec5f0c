// Time mixing: a linear recurrence with a decay per head and key channel that the token chooses, read out before its update with a bonus
// for the current token (ops/recurrence.py):
//
//   o_t = (S_{t-1} + diag(u) k_t v_t^T)^T r_t,   S_t = diag(w_t) S_{t-1} + k_t v_t^T,   log w = -exp(z + w0)
//
//   time_mix_scan        decode rows, short spans, float32: linear_scan.cuh with the decay in the front
//   tanh_rows            the decay projection's activation
#define STK_PDL_CLASS 16
#include "chunk_mma.cuh"
#include "linear_scan.cuh"

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
