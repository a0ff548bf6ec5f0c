// Mixture-of-experts feed-forward with ungated experts, y = W_down relu(W_up x)^2, weights in the compute type (bf16 or fp32).
//
//   expert_rows      one CTA per (pair, block of output rows): a warp streams whole weight rows and dots them with the pair's
//                    activations, fp32 accumulation.  Decode-sized batches, and every batch of a float32 model.
// A pair is one (token, chosen expert).  The weighted sum over a token's pairs is formed where it is normed (hybrid_block.cu).
#define STK_PDL_CLASS 1024
#include "common.cuh"

namespace stk {

template <typename A> struct Vec16;
template <> struct Vec16<float> {
  static constexpr int kN = 4;
  static __device__ __forceinline__ void load(const float* p, float (&f)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    f[0] = v.x; f[1] = v.y; f[2] = v.z; f[3] = v.w;
  }
  static __device__ __forceinline__ float round(float v) { return v; }
};
template <> struct Vec16<__nv_bfloat16> {
  static constexpr int kN = 8;
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[8]) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 u = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&v)[j]);
      f[2 * j] = u.x; f[2 * j + 1] = u.y;
    }
  }
  static __device__ __forceinline__ __nv_bfloat16 round(float v) { return __float2bfloat16(v); }
};

constexpr int kRowsPerWarp = 4, kExpertWarps = 8;

// out[pair, n] = act(x[pair / div] . W[expert(pair), n]) for n < N, zeros up to n_pad.  act: relu squared when `square`.
template <typename A>
__global__ void __launch_bounds__(kExpertWarps * 32)
expert_rows_kernel(const A* __restrict__ x, long long ldx, int div, const A* __restrict__ W, long long estride,
                   const int* __restrict__ ids, int E, A* __restrict__ out, long long ldo, int N, int n_pad, int K, int square) {
  using V = Vec16<A>;
  pdl_wait();
  pdl_trigger();
  const long long pair = blockIdx.y;
  const int e = ids[pair];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = (blockIdx.x * kExpertWarps + warp) * kRowsPerWarp;
  if (n0 >= n_pad) return;
  const bool ok = e >= 0 && e < E;
  const A* xr = x + pair / div * ldx;
  const A* w = W + static_cast<long long>(ok ? e : 0) * estride;
  float acc[kRowsPerWarp];
#pragma unroll
  for (int r = 0; r < kRowsPerWarp; ++r) acc[r] = 0.f;
  for (int k = lane * V::kN; k < K; k += 32 * V::kN) {
    float xv[V::kN], wv[kRowsPerWarp][V::kN];
#pragma unroll
    for (int r = 0; r < kRowsPerWarp; ++r) V::load(w + static_cast<long long>(min(n0 + r, N - 1)) * K + k, wv[r]);
    V::load(xr + k, xv);
#pragma unroll
    for (int r = 0; r < kRowsPerWarp; ++r)
#pragma unroll
      for (int i = 0; i < V::kN; ++i) acc[r] = fmaf(wv[r][i], xv[i], acc[r]);
  }
#pragma unroll
  for (int r = 0; r < kRowsPerWarp; ++r) {
    float v = warp_sum(acc[r]);
    if (square) v = v > 0.f ? v * v : 0.f;
    if (lane == 0 && n0 + r < n_pad) out[pair * ldo + n0 + r] = V::round(ok && n0 + r < N ? v : 0.f);
  }
}

}  // namespace stk

using namespace stk;

// x rows of K elements (K a multiple of 16 bytes' worth, rows 16-byte aligned), W [E, N, K].
STK_API int stk_expert_rows(const void* x, long long ldx, int div, const void* W, const int* ids, int E, void* out, long long ldo,
                            int N, int n_pad, int K, int square, int fp32, int n_pairs, void* stream) {
  if (n_pairs <= 0) return 0;
  const int v = fp32 ? 4 : 8;
  if (K % v || ldx % v || div < 1 || N < 1 || n_pad < N || E < 1) return -1;
  if ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(W)) & 15) return -1;
  const int bx = (n_pad + kExpertWarps * kRowsPerWarp - 1) / (kExpertWarps * kRowsPerWarp);
  cudaStream_t st = (cudaStream_t)stream;
  // the grid's y extent is bounded: long batches go in slices
  for (int p0 = 0; p0 < n_pairs; p0 += 65520 / div * div) {
    const int n = min(n_pairs - p0, 65520 / div * div);
    if (fp32)
      launch_pdl(expert_rows_kernel<float>, dim3(bx, n), dim3(kExpertWarps * 32), 0, st, (const float*)x + (long long)(p0 / div) * ldx,
                 ldx, div, (const float*)W, (long long)N * K, ids + p0, E, (float*)out + (long long)p0 * ldo, ldo, N, n_pad, K, square);
    else
      launch_pdl(expert_rows_kernel<__nv_bfloat16>, dim3(bx, n), dim3(kExpertWarps * 32), 0, st,
                 (const __nv_bfloat16*)x + (long long)(p0 / div) * ldx, ldx, div, (const __nv_bfloat16*)W, (long long)N * K, ids + p0, E,
                 (__nv_bfloat16*)out + (long long)p0 * ldo, ldo, N, n_pad, K, square);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
