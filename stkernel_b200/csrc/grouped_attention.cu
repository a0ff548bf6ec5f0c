// What grouped-query attention over the full context does between its projections and its scores: biases, unit-RMS queries and
// keys, the query temperature, and the insertion of the tokens' rows into the paged cache.  (Scores and outputs:
// window_attention.cu for decode rows, short spans and float32; latent_prompt_tc.cu for long spans.)
//
// A cached row is [value (V) | zeros up to k_col | key (D) | zeros up to `row`], pages are [G][64][row].
#define STK_PDL_CLASS 8
#include "hybrid_block.cuh"

namespace stk {

constexpr int kGqPage = 64, kGqWarps = 8;

struct GqArgs {
  const void* proj; long long ldp; int q_off, k_off, v_off;
  const float* bias;                                   // [H * D | G * D | G * V] or nullptr
  int norm; float eps, coef; double every;
  const int64_t* positions; const int* tok_req;
  const int* table; int bt_stride;
  void* cache; int row, k_col;
  int H, G, D, V;
  void* q; int dp;                                     // queries: head h at columns h * dp, zeros behind D
  int T;
};

// dst[0 : n) = (src + bias) * f, zeros up to n_pad; four elements per lane and pass where everything is aligned.
template <typename A>
__device__ __forceinline__ void gq_store(A* dst, const A* src, const float* bias, int n, int n_pad, float f, bool vec, int lane) {
  if (sizeof(A) == 2 && vec) {
    for (int i = lane * 4; i < n_pad; i += 128) {
      uint2 v = make_uint2(0, 0);
      if (i < n) {
        const uint2 u = *reinterpret_cast<const uint2*>(src + i);
        float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
        float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
        if (bias != nullptr) { a.x += bias[i]; a.y += bias[i + 1]; b.x += bias[i + 2]; b.y += bias[i + 3]; }
        *reinterpret_cast<__nv_bfloat162*>(&v.x) = __floats2bfloat162_rn(a.x * f, a.y * f);
        *reinterpret_cast<__nv_bfloat162*>(&v.y) = __floats2bfloat162_rn(b.x * f, b.y * f);
      }
      *reinterpret_cast<uint2*>(dst + i) = v;
    }
    return;
  }
  for (int i = lane; i < n_pad; i += 32) st_act(dst + i, i < n ? (ld_act(src + i) + (bias != nullptr ? bias[i] : 0.f)) * f : 0.f);
}

template <typename A>
__device__ __forceinline__ float gq_inv_rms(const A* src, const float* bias, int n, float eps, bool vec, int lane) {
  float s = 0.f;
  if (sizeof(A) == 2 && vec) {
    for (int i = lane * 4; i < n; i += 128) {
      const uint2 u = *reinterpret_cast<const uint2*>(src + i);
      float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
      float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
      if (bias != nullptr) { a.x += bias[i]; a.y += bias[i + 1]; b.x += bias[i + 2]; b.y += bias[i + 3]; }
      s = fmaf(a.x, a.x, fmaf(a.y, a.y, fmaf(b.x, b.x, fmaf(b.y, b.y, s))));
    }
  } else {
    for (int i = lane; i < n; i += 32) {
      const float x = ld_act(src + i) + (bias != nullptr ? bias[i] : 0.f);
      s = fmaf(x, x, s);
    }
  }
  return 1.f / sqrtf(warp_sum(s) / static_cast<float>(n) + eps);
}

// One warp per (token, query head or key/value head).
template <typename A>
__global__ void __launch_bounds__(kGqWarps * 32)
grouped_prep_kernel(const GqArgs a, int vec_in, int vec_row) {
  pdl_wait();
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, units = a.H + a.G;
  const long long u = blockIdx.x * static_cast<long long>(kGqWarps) + warp;
  const long long t = u / units;
  if (t >= a.T) return;
  const int unit = static_cast<int>(u - t * units);
  const A* p = reinterpret_cast<const A*>(a.proj) + t * a.ldp;
  const int req = a.tok_req[t];
  const long long pos = a.positions[t];
  const bool live = req >= 0 && pos >= 0;
  if (unit < a.H) {
    const A* src = p + a.q_off + unit * a.D;
    const float* bias = a.bias != nullptr ? a.bias + unit * a.D : nullptr;
    A* dst = reinterpret_cast<A*>(a.q) + (t * a.H + unit) * a.dp;
    if (!live) {
      for (int i = lane; i < a.dp; i += 32) st_act(dst + i, 0.f);
      return;
    }
    float f = a.norm ? gq_inv_rms(src, bias, a.D, a.eps, vec_in, lane) : 1.f;
    if (a.coef != 0.f) f *= 1.f + a.coef * logf(static_cast<float>(floor(static_cast<double>(pos + 1) / a.every)) + 1.f);
    gq_store(dst, src, bias, a.D, a.dp, f, vec_in, lane);
    return;
  }
  if (!live) return;
  const int page = a.table[static_cast<long long>(req) * a.bt_stride + pos / kGqPage];
  if (page < 0) return;
  const int g = unit - a.H;
  A* row = reinterpret_cast<A*>(a.cache) + ((static_cast<long long>(page) * a.G + g) * kGqPage + pos % kGqPage) * a.row;
  const A* k = p + a.k_off + g * a.D;
  const A* v = p + a.v_off + g * a.V;
  const float* kb = a.bias != nullptr ? a.bias + (a.H + g) * a.D : nullptr;
  const float* vb = a.bias != nullptr ? a.bias + (a.H + a.G) * a.D + g * a.V : nullptr;
  gq_store(row, v, vb, a.V, a.k_col, 1.f, vec_row, lane);
  gq_store(row + a.k_col, k, kb, a.D, a.row - a.k_col, a.norm ? gq_inv_rms(k, kb, a.D, a.eps, vec_in, lane) : 1.f, vec_row, lane);
}

}  // namespace stk

using namespace stk;

STK_API int stk_grouped_prep(const void* proj, long long ldp, int q_off, int k_off, int v_off, const float* bias, int norm, float eps,
                             float coef, float every, const int64_t* positions, const int* tok_req, const int* table, int bt_stride,
                             void* cache, int row, int k_col, int heads, int kv_heads, int dim, int vdim, void* q, int dp, int fp32,
                             int T, void* stream) {
  if (T <= 0) return 0;
  if (heads < 1 || kv_heads < 1 || heads % kv_heads || dim < 1 || vdim < 1 || k_col < vdim || row < k_col + dim || dp < dim || every <= 0.f)
    return -1;
  GqArgs a;
  a.proj = proj; a.ldp = ldp; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off;
  a.bias = bias; a.norm = norm; a.eps = eps; a.coef = coef; a.every = every;
  a.positions = positions; a.tok_req = tok_req; a.table = table; a.bt_stride = bt_stride;
  a.cache = cache; a.row = row; a.k_col = k_col;
  a.H = heads; a.G = kv_heads; a.D = dim; a.V = vdim;
  a.q = q; a.dp = dp; a.T = T;
  const uintptr_t at = reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache);
  const int vec_in = !fp32 && dim % 4 == 0 && dp % 4 == 0 && ldp % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && (at & 7) == 0;
  const int vec_row = vec_in && vdim % 4 == 0 && v_off % 4 == 0 && k_col % 4 == 0 && row % 4 == 0;
  const long long warps = static_cast<long long>(T) * (heads + kv_heads);
  const dim3 grid(static_cast<unsigned>((warps + kGqWarps - 1) / kGqWarps));
  cudaStream_t st = (cudaStream_t)stream;
  if (fp32) launch_pdl(grouped_prep_kernel<float>, grid, dim3(kGqWarps * 32), 0, st, a, vec_in, vec_row);
  else launch_pdl(grouped_prep_kernel<__nv_bfloat16>, grid, dim3(kGqWarps * 32), 0, st, a, vec_in, vec_row);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
