// Mixture-of-experts feed-forward, y = W_down act(W_up x) with act relu squared or the exact gelu, or y = W_down (silu(W_gate x) * W_up x)
// with the rows of W_gate and W_up in turns (so that one tile has both); weights in the compute type (bf16 or fp32).
//
//   expert_rows      one CTA per (pair, block of output rows): a warp streams whole weight rows and dots them with the pair's
//                    activations, fp32 accumulation.  A handful of pairs, and every batch of a float32 model.
//   experts_slim     tcgen05, pairs sorted by expert: 128 weight rows x 16..64 tokens per tile (few tokens per expert: the
//                    time is that of streaming the weights)
//   experts_wide     tcgen05, pairs sorted by expert: 256 tokens (two accumulators that share the weight tile; one when the
//                    expert has no more than 128 left) x 256 weight rows
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

constexpr int kActGated = 3;                     // N weight rows give N / 2 results

// silu(gate) * up.
__device__ __forceinline__ float expert_glu(float gate, float up) { return gate / (1.f + expf(-gate)) * up; }
__device__ __forceinline__ float expert_glu_fast(float gate, float up) { return __fdividef(gate, 1.f + __expf(-gate)) * up; }

// act 0: none, 1: relu squared, 2: gelu (exact).  kRounded: the result is rounded to bf16, so the gelu's erfc may come from the rational
// approximation 7.1.26 of Abramowitz and Stegun, Handbook of Mathematical Functions (absolute error 1.5e-7).
template <bool kRounded = true>
__device__ __forceinline__ float expert_act(float v, int act) {
  if (act == 1) return v > 0.f ? v * v : 0.f;
  if (act == 2) {
    if (!kRounded) return 0.5f * v * (1.f + erff(v * 0.70710678118654752f));
    const float z = fabsf(v) * 0.70710678118654752f;
    const float t = __fdividef(1.f, fmaf(0.3275911f, z, 1.f));
    const float p = t * fmaf(t, fmaf(t, fmaf(t, fmaf(t, 1.061405429f, -1.453152027f), 1.421413741f), -0.284496736f), 0.254829592f);
    const float half = 0.5f * v * p * __expf(-z * z);       // v erfc(|v| / sqrt 2) / 2
    return v < 0.f ? half : v - half;
  }
  return v;
}

// out[pair, n] = act(x[pair / div] . W[expert(pair), n]) for n < N, zeros up to n_pad.
template <typename A>
__global__ void __launch_bounds__(kExpertWarps * 32)
expert_rows_kernel(const A* __restrict__ x, long long ldx, int div, const A* __restrict__ W, long long estride,
                   const int* __restrict__ ids, int E, A* __restrict__ out, long long ldo, int N, int n_pad, int K, int act) {
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
  if (act == kActGated) {
#pragma unroll
    for (int r = 0; r < kRowsPerWarp; r += 2) {
      const float v = expert_glu(warp_sum(acc[r]), warp_sum(acc[r + 1]));
      if (lane == 0 && n0 + r < n_pad) out[pair * ldo + (n0 + r) / 2] = V::round(ok && n0 + r < N ? v : 0.f);
    }
    return;
  }
#pragma unroll
  for (int r = 0; r < kRowsPerWarp; ++r) {
    float v = warp_sum(acc[r]);
    v = expert_act<sizeof(A) == 2>(v, act);
    if (lane == 0 && n0 + r < n_pad) out[pair * ldo + n0 + r] = V::round(ok && n0 + r < N ? v : 0.f);
  }
}

// ---- pairs sorted by expert ----------------------------------------------------------------------
int make_tmap_2d(CUtensorMap* tm, const void* base, int elem_bytes, long long rows, long long cols, long long ld, int box_rows);

// sorted row q <- activations of token sorted[q] / topk
__global__ void __launch_bounds__(128)
expert_gather_kernel(const __nv_bfloat16* __restrict__ x, long long ldx, const int* __restrict__ sorted, int topk,
                     __nv_bfloat16* __restrict__ xs, int K) {
  pdl_wait();
  pdl_trigger();
  const long long q = blockIdx.x;
  const uint4* src = reinterpret_cast<const uint4*>(x + static_cast<long long>(sorted[q] / topk) * ldx);
  uint4* dst = reinterpret_cast<uint4*>(xs + q * K);
  for (int i = threadIdx.x; i < K / 8; i += blockDim.x) dst[i] = src[i];
}

struct ExpertArgs {
  const int* offsets;      // [E + 1] first sorted row of every expert
  int E, N, k_blocks, tiles_n;
  __nv_bfloat16* out;      // [P, ldo]
  long long ldo;
  int act;
  int* status;
};
constexpr int kMaxExperts = 512;

struct alignas(8) ExpertBars {
  uint64_t full[8], empty[8], tmem_full[2], tmem_empty[2];
  uint32_t tmem_base;
};

// first[e]: tiles of the experts before e, for tiles of `rows` tokens (first[E] = all tiles).
__device__ __forceinline__ void expert_tiles(int* first, const int* offsets, int E, int rows, int tiles_n) {
  if (threadIdx.x < 32) {
    int run = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + threadIdx.x;
      const int n = e < E ? (offsets[e + 1] - offsets[e] + rows - 1) / rows * tiles_n : 0;
      int incl = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, incl, o);
        if (static_cast<int>(threadIdx.x) >= o) incl += v;
      }
      if (e < E) first[e] = run + incl - n;
      run += __shfl_sync(0xffffffffu, incl, 31);
    }
    if (threadIdx.x == 0) first[E] = run;
  }
}

__device__ __forceinline__ uint32_t expert_pack(uint32_t a, uint32_t b, int act) {
  const float x = expert_act(__uint_as_float(a), act), y = expert_act(__uint_as_float(b), act);
  const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
  return *reinterpret_cast<const uint32_t*>(&v);
}

template <int BT>
struct SlimCfg {
  static constexpr int kStageBytes = 128 * 128 + BT * 128;
  static constexpr int kStages = 8;
  static constexpr int kTmemCols = 2 * BT <= 32 ? 32 : 2 * BT <= 64 ? 64 : 128;
};

template <int BT>
__global__ void __launch_bounds__(192, 1)
experts_slim_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x, const ExpertArgs a) {
  using Cfg = SlimCfg<BT>;
  constexpr int kStages = Cfg::kStages;
  extern __shared__ uint8_t smem_raw[];
  __shared__ int first[kMaxExperts + 1];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* smem_b = smem + kStages * 128 * 128;
  ExpertBars* bars = reinterpret_cast<ExpertBars*>(smem_b + kStages * BT * 128);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 64) {
    for (int s = 0; s < kStages; ++s) {
      mbar_init(&bars->full[s], 1);
      mbar_init(&bars->empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bars->tmem_full[i], 1);
      mbar_init(&bars->tmem_empty[i], 4);
    }
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(&bars->tmem_base, Cfg::kTmemCols);
    tmem_relinquish();
  }
  pdl_wait();
  pdl_trigger();
  expert_tiles(first, a.offsets, a.E, BT, a.tiles_n);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_base;
  const int units = first[a.E];
  if (warp == 0) {
    if (lane == 0) {
      int seq = 0, e = 0;
      bool ok = true;
      for (int u = blockIdx.x; u < units && ok; u += gridDim.x) {
        while (u >= first[e + 1]) ++e;
        const int r = u - first[e], tt = r / a.tiles_n, tn = r - tt * a.tiles_n;
        for (int kb = 0; kb < a.k_blocks; ++kb, ++seq) {
          const int st = seq % kStages;
          if (!mbar_wait(&bars->empty[st], ((seq / kStages) & 1) ^ 1, a.status, 940)) { ok = false; break; }
          mbar_expect_tx(&bars->full[st], Cfg::kStageBytes);
          tma_load_2d(smem + st * 128 * 128, &tm_w, &bars->full[st], kb * 64, e * a.N + tn * 128);
          tma_load_2d(smem_b + st * BT * 128, &tm_x, &bars->full[st], kb * 64, a.offsets[e] + tt * BT);
        }
      }
      if (!ok)
        for (int s = max(0, seq - kStages); s < seq; ++s) mbar_wait(&bars->full[s % kStages], (s / kStages) & 1, nullptr, 0);
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t kIdesc = umma_idesc(1u, 1u, 128, BT);
      int seq = 0, i = 0;
      bool ok = true;
      for (int u = blockIdx.x; u < units && ok; u += gridDim.x, ++i) {
        if (!mbar_wait(&bars->tmem_empty[i & 1], ((i >> 1) & 1) ^ 1, a.status, 941)) break;
        tc_fence_after();
        for (int kb = 0; kb < a.k_blocks; ++kb, ++seq) {
          const int st = seq % kStages;
          if (!mbar_wait(&bars->full[st], (seq / kStages) & 1, a.status, 942)) { ok = false; break; }
          tc_fence_after();
          const uint64_t ad = umma_desc_sw128(smem_u32(smem + st * 128 * 128));
          const uint64_t bd = umma_desc_sw128(smem_u32(smem_b + st * BT * 128));
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_f16(tmem + (i & 1) * BT, ad + 2 * k, bd + 2 * k, kIdesc, (kb > 0 || k > 0) ? 1u : 0u);
          umma_commit(&bars->empty[st]);
        }
        if (ok) umma_commit(&bars->tmem_full[i & 1]);
      }
    }
  } else {
    const int q = warp & 3;
    int i = 0, e = 0;
    for (int u = blockIdx.x; u < units; u += gridDim.x, ++i) {
      while (u >= first[e + 1]) ++e;
      const int r = u - first[e], tt = r / a.tiles_n, tn = r - tt * a.tiles_n;
      if (!mbar_wait(&bars->tmem_full[i & 1], (i >> 1) & 1, a.status, 943)) break;
      tc_fence_after();
      const int n = tn * 128 + q * 32 + lane, valid = min(BT, a.offsets[e + 1] - a.offsets[e] - tt * BT);
      __nv_bfloat16* o = a.out + (static_cast<long long>(a.offsets[e]) + tt * BT) * a.ldo + n;
#pragma unroll
      for (int c = 0; c < BT; c += 16) {
        uint32_t v[16];
        tmem_ld_32x16(tmem + (i & 1) * BT + c + (static_cast<uint32_t>(q * 32) << 16), v);
        tmem_ld_wait();
        if (a.act == kActGated) {
          // an odd lane's row is the value that belongs to the gate of the lane before it
          __nv_bfloat16* og = a.out + (static_cast<long long>(a.offsets[e]) + tt * BT) * a.ldo + (n >> 1);
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const float up = __shfl_down_sync(0xffffffffu, __uint_as_float(v[j]), 1);
            if ((lane & 1) == 0 && n < a.N && c + j < valid) og[(c + j) * a.ldo] = __float2bfloat16(expert_glu_fast(__uint_as_float(v[j]), up));
          }
        } else if (n < a.N) {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (c + j < valid) o[(c + j) * a.ldo] = __float2bfloat16(expert_act(__uint_as_float(v[j]), a.act));
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->tmem_empty[i & 1]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, Cfg::kTmemCols);
  }
}

constexpr int kXwStages = 3, kXwStageBytes = 2 * 128 * 128 + 256 * 128;

__global__ void __launch_bounds__(320, 1)
experts_wide_kernel(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x, const ExpertArgs a) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ int first[kMaxExperts + 1];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  ExpertBars* bars = reinterpret_cast<ExpertBars*>(smem + kXwStages * kXwStageBytes);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 64) {
    for (int s = 0; s < kXwStages; ++s) {
      mbar_init(&bars->full[s], 1);
      mbar_init(&bars->empty[s], 1);
    }
    mbar_init(&bars->tmem_full[0], 1);
    mbar_init(&bars->tmem_empty[0], 8);
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc(&bars->tmem_base, 512);
    tmem_relinquish();
  }
  pdl_wait();
  pdl_trigger();
  expert_tiles(first, a.offsets, a.E, 256, a.tiles_n);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = bars->tmem_base;
  const int units = first[a.E];
  if (warp == 0) {
    if (lane == 0) {
      int seq = 0, e = 0;
      bool ok = true;
      for (int u = blockIdx.x; u < units && ok; u += gridDim.x) {
        while (u >= first[e + 1]) ++e;
        const int r = u - first[e], tt = r / a.tiles_n, tn = r - tt * a.tiles_n;
        const int row = a.offsets[e] + tt * 256;
        const bool two = a.offsets[e + 1] - row > 128;
        for (int kb = 0; kb < a.k_blocks; ++kb, ++seq) {
          const int st = seq % kXwStages;
          if (!mbar_wait(&bars->empty[st], ((seq / kXwStages) & 1) ^ 1, a.status, 950)) { ok = false; break; }
          mbar_expect_tx(&bars->full[st], kXwStageBytes - (two ? 0 : 128 * 128));
          uint8_t* s = smem + st * kXwStageBytes;
          tma_load_2d(s, &tm_x, &bars->full[st], kb * 64, row);
          if (two) tma_load_2d(s + 128 * 128, &tm_x, &bars->full[st], kb * 64, row + 128);
          tma_load_2d(s + 2 * 128 * 128, &tm_w, &bars->full[st], kb * 64, e * a.N + tn * 256);
        }
      }
      if (!ok)
        for (int s = max(0, seq - kXwStages); s < seq; ++s) mbar_wait(&bars->full[s % kXwStages], (s / kXwStages) & 1, nullptr, 0);
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t kIdesc = umma_idesc(1u, 1u, 128, 256);
      int seq = 0, i = 0, e = 0;
      bool ok = true;
      for (int u = blockIdx.x; u < units && ok; u += gridDim.x, ++i) {
        while (u >= first[e + 1]) ++e;
        const bool two = a.offsets[e + 1] - a.offsets[e] - (u - first[e]) / a.tiles_n * 256 > 128;
        if (!mbar_wait(&bars->tmem_empty[0], (i & 1) ^ 1, a.status, 951)) break;
        tc_fence_after();
        for (int kb = 0; kb < a.k_blocks; ++kb, ++seq) {
          const int st = seq % kXwStages;
          if (!mbar_wait(&bars->full[st], (seq / kXwStages) & 1, a.status, 952)) { ok = false; break; }
          tc_fence_after();
          const uint8_t* s = smem + st * kXwStageBytes;
          const uint64_t a0 = umma_desc_sw128(smem_u32(s)), a1 = umma_desc_sw128(smem_u32(s + 128 * 128));
          const uint64_t bd = umma_desc_sw128(smem_u32(s + 2 * 128 * 128));
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const uint32_t acc = (kb > 0 || k > 0) ? 1u : 0u;
            umma_f16(tmem, a0 + 2 * k, bd + 2 * k, kIdesc, acc);
            if (two) umma_f16(tmem + 256, a1 + 2 * k, bd + 2 * k, kIdesc, acc);
          }
          umma_commit(&bars->empty[st]);
        }
        if (ok) umma_commit(&bars->tmem_full[0]);
      }
    }
  } else {
    const int q = warp & 3, half = (warp - 2) >> 2;                 // the warp's TMEM lanes, its half of the columns
    int i = 0, e = 0;
    for (int u = blockIdx.x; u < units; u += gridDim.x, ++i) {
      while (u >= first[e + 1]) ++e;
      const int r = u - first[e], tt = r / a.tiles_n, tn = r - tt * a.tiles_n;
      if (!mbar_wait(&bars->tmem_full[0], i & 1, a.status, 953)) break;
      tc_fence_after();
      const int row0 = a.offsets[e] + tt * 256, left = a.offsets[e + 1] - row0;
      for (int m = 0; m < (left > 128 ? 2 : 1); ++m) {
        const int t = m * 128 + q * 32 + lane;
        __nv_bfloat16* o = a.out + static_cast<long long>(row0 + (t < left ? t : 0)) * a.ldo + tn * 256;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t v[32];
          const int col = half * 128 + c * 32;
          tmem_ld_32x32(tmem + m * 256 + col + (static_cast<uint32_t>(q * 32) << 16), v);
          tmem_ld_wait();
          if (t < left && a.act == kActGated) {
            __nv_bfloat16* og = a.out + static_cast<long long>(row0 + t) * a.ldo + (tn * 256 + col) / 2;
#pragma unroll
            for (int j = 0; j < 32; j += 8)
              if (tn * 256 + col + j < a.N) {
                __align__(8) __nv_bfloat162 b[2];
#pragma unroll
                for (int k = 0; k < 2; ++k)
                  b[k] = __floats2bfloat162_rn(expert_glu_fast(__uint_as_float(v[j + 4 * k]), __uint_as_float(v[j + 4 * k + 1])),
                                               expert_glu_fast(__uint_as_float(v[j + 4 * k + 2]), __uint_as_float(v[j + 4 * k + 3])));
                *reinterpret_cast<uint2*>(og + j / 2) = *reinterpret_cast<const uint2*>(b);
              }
          } else if (t < left) {
#pragma unroll
            for (int j = 0; j < 32; j += 8)
              if (tn * 256 + col + j < a.N)                          // N is a multiple of 8
                *reinterpret_cast<uint4*>(o + col + j) =
                    make_uint4(expert_pack(v[j], v[j + 1], a.act), expert_pack(v[j + 2], v[j + 3], a.act),
                               expert_pack(v[j + 4], v[j + 5], a.act), expert_pack(v[j + 6], v[j + 7], a.act));
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars->tmem_empty[0]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

template <int BT>
static int launch_slim(const CUtensorMap& tw, const CUtensorMap& tx, const ExpertArgs& a, int grid, cudaStream_t st) {
  const int smem = SlimCfg<BT>::kStages * SlimCfg<BT>::kStageBytes + 256 + 1024;
  static_assert(sizeof(ExpertBars) <= 256, "barrier block");
  if (cudaFuncSetAttribute(experts_slim_kernel<BT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
  launch_pdl(experts_slim_kernel<BT>, dim3(grid), dim3(192), smem, st, tw, tx, a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace stk

using namespace stk;

// act 3: `out` has N / 2 columns (n_pad / 2 of them are written), N even.  x rows of K elements (K a multiple of 16 bytes' worth, rows 16-byte aligned), W [E, N, K].
STK_API int stk_expert_rows(const void* x, long long ldx, int div, const void* W, const int* ids, int E, void* out, long long ldo,
                            int N, int n_pad, int K, int act, int fp32, int n_pairs, void* stream) {
  if (n_pairs <= 0) return 0;
  const int v = fp32 ? 4 : 8;
  if (K % v || ldx % v || div < 1 || N < 1 || n_pad < N || E < 1 || (act == kActGated && (N | n_pad) % 2)) return -1;
  if ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(W)) & 15) return -1;
  const int bx = (n_pad + kExpertWarps * kRowsPerWarp - 1) / (kExpertWarps * kRowsPerWarp);
  cudaStream_t st = (cudaStream_t)stream;
  // the grid's y extent is bounded: long batches go in slices
  for (int p0 = 0; p0 < n_pairs; p0 += 65520 / div * div) {
    const int n = min(n_pairs - p0, 65520 / div * div);
    if (fp32)
      launch_pdl(expert_rows_kernel<float>, dim3(bx, n), dim3(kExpertWarps * 32), 0, st, (const float*)x + (long long)(p0 / div) * ldx,
                 ldx, div, (const float*)W, (long long)N * K, ids + p0, E, (float*)out + (long long)p0 * ldo, ldo, N, n_pad, K, act);
    else
      launch_pdl(expert_rows_kernel<__nv_bfloat16>, dim3(bx, n), dim3(kExpertWarps * 32), 0, st,
                 (const __nv_bfloat16*)x + (long long)(p0 / div) * ldx, ldx, div, (const __nv_bfloat16*)W, (long long)N * K, ids + p0, E,
                 (__nv_bfloat16*)out + (long long)p0 * ldo, ldo, N, n_pad, K, act);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_expert_gather(const void* x, long long ldx, const int* sorted, int topk, void* xs, int K, int n_pairs, void* stream) {
  if (n_pairs <= 0) return 0;
  if (K % 8 || ldx % 8 || topk < 1) return -1;
  launch_pdl(expert_gather_kernel, dim3(n_pairs), dim3(128), 0, (cudaStream_t)stream, (const __nv_bfloat16*)x, ldx, sorted, topk,
             (__nv_bfloat16*)xs, K);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// xs [n_pairs, K] sorted by expert, W [E, N, K], out [n_pairs, ldo] (act 3: N / 2 columns); bf16.  The tile follows the average number of pairs an expert has.
STK_API int stk_experts(const void* xs, int n_pairs, const void* W, const int* offsets, int E, int N, int K, void* out, long long ldo,
                        int act, int sm_count, int* status, void* stream) {
  if (n_pairs <= 0) return 0;
  if (E < 1 || E > kMaxExperts || N % 8 || K % 8 || ldo % 8 || static_cast<long long>(E) * N >= (1ll << 31) ||
      ((reinterpret_cast<uintptr_t>(xs) | reinterpret_cast<uintptr_t>(W) | reinterpret_cast<uintptr_t>(out)) & 15))
    return -1;
  const int avg = n_pairs / E;
  const bool wide = avg > 64 && N >= 128;
  const int bt = avg <= 8 ? 16 : avg <= 24 ? 32 : 64;
  CUtensorMap tw, tx;
  if (make_tmap_2d(&tw, W, 2, static_cast<long long>(E) * N, K, K, wide ? 256 : 128) != 0) return -2;
  if (make_tmap_2d(&tx, xs, 2, n_pairs, K, K, wide ? 128 : bt) != 0) return -2;
  ExpertArgs a;
  a.offsets = offsets; a.E = E; a.N = N; a.k_blocks = (K + 63) / 64; a.tiles_n = wide ? (N + 255) / 256 : (N + 127) / 128;
  a.out = (__nv_bfloat16*)out; a.ldo = ldo; a.act = act; a.status = status;
  cudaStream_t st = (cudaStream_t)stream;
  // no more CTAs than there can be tiles
  const int rows = wide ? 256 : bt;
  const long long most = (static_cast<long long>(n_pairs) / rows + (n_pairs < E ? n_pairs : E)) * a.tiles_n;
  const int grid = most < sm_count ? static_cast<int>(most) : sm_count;
  if (wide) {
    const int smem = kXwStages * kXwStageBytes + 256 + 1024;
    if (cudaFuncSetAttribute(experts_wide_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -3;
    launch_pdl(experts_wide_kernel, dim3(grid), dim3(320), smem, st, tw, tx, a);
    return cudaGetLastError() == cudaSuccess ? 0 : -4;
  }
  switch (bt) {
    case 16: return launch_slim<16>(tw, tx, a, grid, st);
    case 32: return launch_slim<32>(tw, tx, a, grid, st);
    default: return launch_slim<64>(tw, tx, a, grid, st);
  }
}
