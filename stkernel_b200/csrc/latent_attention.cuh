// Arguments and small helpers shared by the latent-attention kernels (latent_attention.cu, latent_attention_tc.cu).
//
// A cached row holds the normed latent in columns [0, C), zeros up to `rot_off`, and the rotated key part that all heads share
// in columns [rot_off, rot_off + R), zeros to the end of the row.
#pragma once
#include "common.cuh"

namespace stk {

constexpr int kLatPage = 64;

struct LatArgs {
  const void* qa; long long ldqa; int cp;         // queries in latent space: head h at columns h * cp
  const void* qr; long long ldqr;                 // rotated query parts before rotation: head h at columns h * R
  const float* gate; long long ldg;               // output-gate logits, one per head (nullptr: no gate)
  const int64_t* positions; const int* tok_req;
  const int* table; int bt_stride;
  const void* cache; int row, rot_off;
  const float* freq;                              // [2][R / 2]: radians per position, high parts then remainders
  int H, C, R;
  float scale;
  void* out; long long ldo;                       // latent read-outs: head h at columns h * cp
};

// cos and sin of position * (hi + lo): the product's rounding error and the frequency's remainder, a small angle together, are
// added by the angle-sum formulas, so the result is good to 32-bit resolution however far the position is.
__device__ __forceinline__ float2 lat_cos_sin(long long pos, float hi, float lo) {
  const float p = static_cast<float>(pos);
  const float a = p * hi;
  const float e = fmaf(p, hi, -a) + p * lo;
  float s, c;
  sincosf(a, &s, &c);
  const float e2 = e * e;
  const float se = fmaf(-e * e2, 1.f / 6.f, e), ce = fmaf(e2, fmaf(e2, 1.f / 24.f, -0.5f), 1.f);
  return make_float2(c * ce - s * se, s * ce + c * se);
}

__device__ __forceinline__ float lat_f(float v) { return v; }
__device__ __forceinline__ float lat_f(__nv_bfloat16 v) { return bf16_to_f(v); }
__device__ __forceinline__ void lat_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void lat_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float lat_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

}  // namespace stk

static inline stk::LatArgs lat_args(const void* qa, long long ldqa, int cp, const void* qr, long long ldqr, const float* gate,
                                    long long ldg, const int64_t* positions, const int* tok_req, const int* table, int bt_stride,
                                    const void* cache, int row, int rot_off, const float* freq, int heads, int kv_rank, int rot,
                                    float scale, void* out, long long ldo) {
  stk::LatArgs a;
  a.qa = qa; a.ldqa = ldqa; a.cp = cp; a.qr = qr; a.ldqr = ldqr; a.gate = gate; a.ldg = ldg;
  a.positions = positions; a.tok_req = tok_req; a.table = table; a.bt_stride = bt_stride;
  a.cache = cache; a.row = row; a.rot_off = rot_off; a.freq = freq;
  a.H = heads; a.C = kv_rank; a.R = rot; a.scale = scale; a.out = out; a.ldo = ldo;
  return a;
}
static inline bool lat_ok(const stk::LatArgs& a) {
  return a.H > 0 && a.C > 0 && a.R >= 0 && (a.R & 1) == 0 && a.cp >= a.C && a.rot_off >= a.C && a.row >= a.rot_off + a.R &&
         a.row <= 2304;
}
