// Arguments and small helpers shared by the windowed-attention kernels (window_attention.cu, window_attention_tc.cu).
#pragma once
#include "common.cuh"

namespace stk {

constexpr int kPage = 64;

struct WinArgs {
  const void* proj; long long ldp; int q_off, k_off;
  const int64_t* positions; const int* tok_req;
  const int* table; int bt_stride;
  void* cache; int row;
  const float* freq; int rd; float mag;
  int H, G, D;
  int window; float scale, softcap; const float* sink;
  void* out; long long ldo;
  // rows of another layout: [value (V columns) .. | key from column k_col on], queries given as they enter the scores (rd = 0)
  int k_col, V, q_step;                           // q_step: columns between the queries of neighbouring heads
  const void* gate; long long ldg;                // output gate logits, [T, H * V] (nullptr: none)
  float out_scale;
};

constexpr float kLog2e = 1.4426950408889634f;
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// Factor on column c of head h's output: out_scale, times the sigmoid of its gate logit if there is a gate.
template <typename A>
__device__ __forceinline__ float win_factor(const WinArgs& a, long long t, int h, int c) {
  if (a.gate == nullptr) return a.out_scale;
  const float z = static_cast<float>(reinterpret_cast<const A*>(a.gate)[t * a.ldg + h * a.V + c]);
  return a.out_scale / (1.f + expf(-z));
}

}  // namespace stk

static inline stk::WinArgs win_args(const void* proj, long long ldp, int q_off, int k_off, const int64_t* positions, const int* tok_req,
                        const int* table, int bt_stride, void* cache, int row, const float* freq, int rd, float mag, int heads,
                        int kv_heads, int dim, int window = 0, float scale = 0.f, float softcap = 0.f,
                        const float* sink = nullptr, void* out = nullptr, long long ldo = 0) {
  stk::WinArgs a;
  a.proj = proj; a.ldp = ldp; a.q_off = q_off; a.k_off = k_off;
  a.positions = positions; a.tok_req = tok_req;
  a.table = table; a.bt_stride = bt_stride;
  a.cache = cache; a.row = row;
  a.freq = freq; a.rd = rd; a.mag = mag;
  a.H = heads; a.G = kv_heads; a.D = dim;
  a.window = window; a.scale = scale; a.softcap = softcap; a.sink = sink;
  a.out = out; a.ldo = ldo;
  a.k_col = rd; a.V = dim; a.q_step = dim;
  a.gate = nullptr; a.ldg = 0; a.out_scale = 1.f;
  return a;
}
static inline void win_layout(stk::WinArgs& a, int k_col, int vdim, int q_step, const void* gate, long long ldg, float out_scale) {
  a.k_col = k_col; a.V = vdim; a.q_step = q_step;
  a.gate = gate; a.ldg = ldg; a.out_scale = out_scale;
}
static inline bool win_ok(const stk::WinArgs& a) {
  return a.H > 0 && a.G > 0 && a.D > 0 && a.H % a.G == 0 && a.rd >= 0 && (a.rd & 1) == 0 && a.rd <= a.D && a.D <= 1024 &&
         a.V > 0 && a.V <= 1024 && a.row >= a.k_col + a.D && a.row >= a.V && a.q_step >= a.D &&
         (a.rd > 0 || a.k_col == 0 || a.k_col >= a.V) && (a.rd == 0 || (a.k_col == a.rd && a.V == a.D && a.row >= a.D + a.rd));
}
// tensor-core kernels: whole 16-byte rows, head size within the accumulators
static inline bool win_mma_ok(const stk::WinArgs& a) {
  return win_ok(a) && a.D <= 256 && a.V <= 256 && a.row % 8 == 0 && (a.rd > 0 || a.k_col % 16 == 0) &&
         (reinterpret_cast<uintptr_t>(a.cache) & 15) == 0;
}
