// Arguments and small helpers shared by the talking-heads attention kernels (talking_attention.cu, talking_tokens_tc.cu,
// talking_prompt_tc.cu).
#pragma once
#include "common.cuh"

namespace stk {

constexpr int kTkPage = 64;

struct TalkArgs {
  const void* q; int T;                           // mixed queries [H, T, G * kp]
  const float* gate; const float* sink;           // [T, H] gate logits, [H] scores without a key (nullptr: none)
  const int64_t* positions; const int* tok_req;
  const int* table; int bt_stride;
  const void* cache; int row, k_col, kp, vp;
  int H, G, V;
  int chunk;                                      // 0: the full context
  float scale;
  void* out; long long ldo; int out_cols;         // head h at columns h * V, zeros behind the last one
};

// First key that a position sees.
__device__ __forceinline__ int talk_first(const TalkArgs& a, long long pos) {
  const int p = static_cast<int>(pos);
  return a.chunk > 0 ? p / a.chunk * a.chunk : 0;
}
__device__ __forceinline__ float talk_gate(const TalkArgs& a, long long t, int h) {
  return a.gate != nullptr ? 1.f / (1.f + expf(-a.gate[t * a.H + h])) : 1.f;
}

}  // namespace stk

static inline bool talk_ok(const stk::TalkArgs& a) {
  return a.H > 0 && a.G > 0 && a.H % a.G == 0 && a.V > 0 && a.vp >= a.V && a.kp > 0 && a.k_col == a.G * a.vp && a.chunk >= 0 &&
         a.row >= a.k_col + a.G * a.kp && a.out_cols >= a.H * a.V;
}
