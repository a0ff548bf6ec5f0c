// Arguments and small helpers shared by the latent-attention kernels (latent_attention.cu, latent_attention_tc.cu).
//
// A cached row holds the normed latent in columns [0, C), zeros up to `rot_off`, and the rotated key part that all heads share
// in columns [rot_off, rot_off + R), zeros to the end of the row.
#pragma once
#include "common.cuh"
#include "pairs.cuh"

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

__device__ __forceinline__ float lat_f(float v) { return v; }
__device__ __forceinline__ float lat_f(__nv_bfloat16 v) { return bf16_to_f(v); }
__device__ __forceinline__ void lat_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void lat_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float lat_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }


// ---- issue of tensor-core products by a converged warp -----------------------------------------------
// The whole warp runs the issuing code with warp-uniform operands (descriptors are their low words; the high word is the same for
// every 128-byte-swizzled operand here) and one elected lane executes the instruction: a few instructions per product, which
// small products need to keep the tensor pipe busy.
constexpr uint32_t kDescHi = (1024u >> 4) | (1u << 14) | (2u << 29);      // 8-row groups 1024 bytes apart, version, 128-byte swizzle
__device__ __forceinline__ uint32_t desc_lo(uint32_t smem_addr, uint32_t lbo_bytes = 16) {
  return ((smem_addr & 0x3FFFF) >> 4) | ((lbo_bytes >> 4) << 16);
}
// D[tmem] (+)= A[smem] * B[smem]
__device__ __forceinline__ void mma_ss(uint32_t d, uint32_t a_lo, uint32_t b_lo, uint32_t idesc, uint32_t acc, uint32_t lead) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t.reg .b64 a, b;\n\t"
      "setp.ne.b32 p, %5, 0;\n\tsetp.ne.b32 q, %6, 0;\n\t"
      "mov.b64 a, {%1, %3};\n\tmov.b64 b, {%2, %3};\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], a, b, %4, p;\n\t}"
      ::"r"(d), "r"(a_lo), "r"(b_lo), "r"(kDescHi), "r"(idesc), "r"(acc), "r"(lead)
      : "memory");
}
// D[tmem] (+)= A[tmem] * B[smem]
__device__ __forceinline__ void mma_ts(uint32_t d, uint32_t a_tmem, uint32_t b_lo, uint32_t idesc, uint32_t acc, uint32_t lead) {
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t.reg .b64 b;\n\t"
      "setp.ne.b32 p, %5, 0;\n\tsetp.ne.b32 q, %6, 0;\n\t"
      "mov.b64 b, {%2, %3};\n\t"
      "@q tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], b, %4, p;\n\t}"
      ::"r"(d), "r"(a_tmem), "r"(b_lo), "r"(kDescHi), "r"(idesc), "r"(acc), "r"(lead)
      : "memory");
}
__device__ __forceinline__ void mma_commit(uint64_t* bar, uint32_t lead) {
  asm volatile(
      "{\n\t.reg .pred q;\n\tsetp.ne.b32 q, %1, 0;\n\t"
      "@q tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];\n\t}"
      ::"r"(smem_u32(bar)), "r"(lead) : "memory");
}

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
