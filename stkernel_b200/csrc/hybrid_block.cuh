// The feed-forward half of the joined sublayer buffer (models/hybrid.py), shared by the kernels that form it.
#pragma once
#include "common.cuh"

namespace stk {

template <typename T> __device__ __forceinline__ float ld_act(const T* p);
template <> __device__ __forceinline__ float ld_act<float>(const float* p) { return *p; }
template <> __device__ __forceinline__ float ld_act<__nv_bfloat16>(const __nv_bfloat16* p) { return bf16_to_f(*p); }
template <typename T> __device__ __forceinline__ void st_act(T* p, float v);
template <> __device__ __forceinline__ void st_act<float>(float* p, float v) { *p = v; }
template <> __device__ __forceinline__ void st_act<__nv_bfloat16>(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// x sigmoid(x) for results that are rounded to bf16: one exponential and one reciprocal of the special-function unit.
__device__ __forceinline__ float silu_bf16(float x) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * -1.4426950408889634f));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
  return x * r;
}

// o[j] = act(gate_j) * up_j for j < ff, zero for ff <= j < n: the eight columns from `base` on.  vec: 16-byte accesses allowed.
// relu: act is relu, else silu.
template <typename A>
__device__ __forceinline__ void glu_columns(const A* pg, const A* pu, A* o, int base, int ff, int n, bool vec,
                                            int relu = 0) {
  if (base >= n) return;
  if (sizeof(A) == 2 && base + 8 <= ff && vec) {
    const uint4 gv = *reinterpret_cast<const uint4*>(pg + base), uv = *reinterpret_cast<const uint4*>(pu + base);
    const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&gv);
    const __nv_bfloat162* u2 = reinterpret_cast<const __nv_bfloat162*>(&uv);
    uint4 ov;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&ov);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 g = __bfloat1622float2(g2[j]), u = __bfloat1622float2(u2[j]);
      o2[j] = relu ? __floats2bfloat162_rn(fmaxf(g.x, 0.f) * u.x, fmaxf(g.y, 0.f) * u.y)
                   : __floats2bfloat162_rn(g.x / (1.f + __expf(-g.x)) * u.x, g.y / (1.f + __expf(-g.y)) * u.y);
    }
    *reinterpret_cast<uint4*>(o + base) = ov;
    return;
  }
  for (int j = base; j < base + 8 && j < n; ++j) {
    float v = 0.f;
    if (j < ff) {
      const float g = ld_act(pg + j);
      v = (relu ? fmaxf(g, 0.f) : g / (1.f + expf(-g))) * ld_act(pu + j);
    }
    st_act(o + j, v);
  }
}

}  // namespace stk
