// Reductions of many values per lane over a warp (attention kernels whose scores have one key per lane and one query per column).
#pragma once
#include "common.cuh"

namespace stk {

// One level of a butterfly all-lane reduction over CNT values per lane: lanes exchange the half they
// give up, so 32 lanes x CNT values reduce with CNT-ish shuffles instead of 5 x CNT.
template <int CNT, bool kMax>
__device__ __forceinline__ void bfly_level(float* v, int off, bool bit) {
  if constexpr (CNT > 1) {
    constexpr int H = CNT / 2;
#pragma unroll
    for (int i = 0; i < H; ++i) {
      const float mine = bit ? v[H + i] : v[i];
      const float send = bit ? v[i] : v[H + i];
      const float recv = __shfl_xor_sync(0xffffffffu, send, off);
      v[i] = kMax ? fmaxf(mine, recv) : mine + recv;
    }
  } else {
    const float recv = __shfl_xor_sync(0xffffffffu, v[0], off);
    v[0] = kMax ? fmaxf(v[0], recv) : v[0] + recv;
  }
}
// Reduce v[h] over the 32 lanes for every h < NH; lane l ends with heads (l*NH/32) .. +max(NH/32,1)
// in v[0..]; they are written to out[h].
template <int NH, bool kMax>
__device__ __forceinline__ void bfly_reduce_store(float (&v)[NH], float* out, int lane) {
  constexpr int C1 = NH / 2 > 0 ? NH / 2 : 1, C2 = C1 / 2 > 0 ? C1 / 2 : 1, C3 = C2 / 2 > 0 ? C2 / 2 : 1,
                C4 = C3 / 2 > 0 ? C3 / 2 : 1, C5 = C4 / 2 > 0 ? C4 / 2 : 1;
  bfly_level<NH, kMax>(v, 16, (lane & 16) != 0);
  bfly_level<C1, kMax>(v, 8, (lane & 8) != 0);
  bfly_level<C2, kMax>(v, 4, (lane & 4) != 0);
  bfly_level<C3, kMax>(v, 2, (lane & 2) != 0);
  bfly_level<C4, kMax>(v, 1, (lane & 1) != 0);
  const int base = (lane * NH) >> 5;
#pragma unroll
  for (int i = 0; i < C5; ++i) out[base + i] = v[i];
}

}  // namespace stk
