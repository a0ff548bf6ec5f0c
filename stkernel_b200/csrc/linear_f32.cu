// True fp32 linear layer on the CUDA cores: out[t, n] = sum_k x[t, k] * W[n, k], fp32 operands and accumulation, no
// reduced-precision products.  Models that run in float32 use it for every projection.
//
//   linear_f32_kernel       64 x 64 output tile per CTA, 16 x 16 threads with 4 x 4 outputs each, K in blocks of 16 staged
//                           in shared memory (k-major, so a thread's four operands are one 16-byte read);
//   linear_f32_rows_kernel  at most eight tokens: one warp per weight row, lanes along K.
// Any sizes; rows need no alignment.
#define STK_PDL_CLASS 2
#include "common.cuh"

namespace stk {

constexpr int kF32Tile = 64, kF32K = 16;

__global__ void __launch_bounds__(256)
linear_f32_kernel(const float* __restrict__ W, long long ldw, const float* __restrict__ x, long long ldx,
                  float* __restrict__ out, long long ldo, int T, int N, int K) {
  __shared__ __align__(16) float xs[kF32K][kF32Tile + 4];
  __shared__ __align__(16) float ws[kF32K][kF32Tile + 4];
  pdl_wait();
  pdl_trigger();
  const int t0 = blockIdx.y * kF32Tile, n0 = blockIdx.x * kF32Tile;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += kF32K) {
    for (int e = threadIdx.x; e < kF32K * kF32Tile; e += 256) {
      const int k = e & (kF32K - 1), r = e / kF32K;
      const bool kin = k0 + k < K;
      xs[k][r] = kin && t0 + r < T ? x[static_cast<long long>(t0 + r) * ldx + k0 + k] : 0.f;
      ws[k][r] = kin && n0 + r < N ? W[static_cast<long long>(n0 + r) * ldw + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kF32K; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + ty * 4 + i;
    if (t >= T) break;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (n0 + tx * 4 + j < N) out[t * ldo + n0 + tx * 4 + j] = acc[i][j];
  }
}

template <int T_>
__global__ void __launch_bounds__(256)
linear_f32_rows_kernel(const float* __restrict__ W, long long ldw, const float* __restrict__ x, long long ldx,
                       float* __restrict__ out, long long ldo, int T, int N, int K) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const int n = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (n >= N) return;
  const float* w = W + n * ldw;
  float acc[T_];
#pragma unroll
  for (int t = 0; t < T_; ++t) acc[t] = 0.f;
  for (int k = lane; k < K; k += 32) {
    const float wv = __ldg(w + k);
#pragma unroll
    for (int t = 0; t < T_; ++t)
      if (t < T) acc[t] = fmaf(wv, x[t * ldx + k], acc[t]);
  }
#pragma unroll
  for (int t = 0; t < T_; ++t) {
    const float v = warp_sum(acc[t]);
    if (lane == 0 && t < T) out[t * ldo + n] = v;
  }
}

}  // namespace stk

using namespace stk;

STK_API int stk_linear_f32(const float* W, long long ldw, const float* x, long long ldx, float* out, long long ldo, int T,
                           int N, int K, void* stream) {
  if (T <= 0 || N <= 0) return 0;
  if (K <= 0) return -1;
  cudaStream_t st = (cudaStream_t)stream;
  if (T <= 8) {
    const dim3 grid((N + 7) / 8);
    if (T == 1)
      launch_pdl(linear_f32_rows_kernel<1>, grid, dim3(256), 0, st, W, ldw, x, ldx, out, ldo, T, N, K);
    else
      launch_pdl(linear_f32_rows_kernel<8>, grid, dim3(256), 0, st, W, ldw, x, ldx, out, ldo, T, N, K);
  } else {
    launch_pdl(linear_f32_kernel, dim3((N + kF32Tile - 1) / kF32Tile, (T + kF32Tile - 1) / kF32Tile), dim3(256), 0, st, W, ldw,
               x, ldx, out, ldo, T, N, K);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
