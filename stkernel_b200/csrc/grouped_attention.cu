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

// bf16 with everything in whole groups of eight: one CTA per token, L lanes per head, eight columns a lane.
template <int L>
__global__ void __launch_bounds__(512)
grouped_prep_vec_kernel(const GqArgs a) {
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const int group = threadIdx.x / L, l = threadIdx.x % L, groups = blockDim.x / L, c = l * 8;
  const int req = a.tok_req[t];
  const long long pos = a.positions[t];
  const bool live = req >= 0 && pos >= 0;
  const int page = live ? a.table[static_cast<long long>(req) * a.bt_stride + pos / kGqPage] : -1;
  const float temp = live && a.coef != 0.f ? 1.f + a.coef * logf(static_cast<float>(floor(static_cast<double>(pos + 1) / a.every)) + 1.f) : 1.f;
  const __nv_bfloat16* p = reinterpret_cast<const __nv_bfloat16*>(a.proj) + t * a.ldp;
  const int units = a.H + 2 * a.G, rounds = (units + groups - 1) / groups;
  for (int i = 0; i < rounds; ++i) {                                  // query heads, key heads, value heads
    const int u = i * groups + group;
    const bool q = u < a.H, k = !q && u < a.H + a.G, ok = u < units;
    const int g = q ? u : k ? u - a.H : u - a.H - a.G, n = q || k ? a.D : a.V;
    float x[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) x[j] = 0.f;
    if (ok && c < n) {
      const uint4 v = *reinterpret_cast<const uint4*>(p + (q ? a.q_off : k ? a.k_off : a.v_off) + g * n + c);
      const float* b = a.bias != nullptr ? a.bias + (q ? 0 : k ? a.H * a.D : (a.H + a.G) * a.D) + g * n + c : nullptr;
      float4 b0 = make_float4(0.f, 0.f, 0.f, 0.f), b1 = b0;
      if (b != nullptr) {
        b0 = *reinterpret_cast<const float4*>(b);
        b1 = *reinterpret_cast<const float4*>(b + 4);
      }
      const float bb[8] = {b0.x, b0.y, b0.z, b0.w, b1.x, b1.y, b1.z, b1.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&v)[j]);
        x[2 * j] = f.x + bb[2 * j];
        x[2 * j + 1] = f.y + bb[2 * j + 1];
      }
    }
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) s = fmaf(x[j], x[j], s);
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    float f = a.norm && (q || k) ? 1.f / sqrtf(s / static_cast<float>(n) + a.eps) : 1.f;
    if (q) f = live ? f * temp : 0.f;
    uint4 r;
#pragma unroll
    for (int j = 0; j < 4; ++j) reinterpret_cast<__nv_bfloat162*>(&r)[j] = __floats2bfloat162_rn(x[2 * j] * f, x[2 * j + 1] * f);
    if (!ok) continue;
    if (q) {
      if (c < a.dp) *reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(a.q) + (t * a.H + g) * a.dp + c) = r;
    } else if (page >= 0) {
      __nv_bfloat16* row = reinterpret_cast<__nv_bfloat16*>(a.cache) + ((static_cast<long long>(page) * a.G + g) * kGqPage + pos % kGqPage) * a.row;
      if (c < (k ? a.row - a.k_col : a.k_col)) *reinterpret_cast<uint4*>(row + (k ? a.k_col : 0) + c) = r;
    }
  }
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
  const int widest = dp > row - k_col ? (dp > k_col ? dp : k_col) : (row - k_col > k_col ? row - k_col : k_col);
  if (!fp32 && (dim | vdim | dp | row | k_col | q_off | k_off | v_off) % 8 == 0 && ldp % 8 == 0 && widest <= 256 &&
      ((at | reinterpret_cast<uintptr_t>(bias)) & 15) == 0) {
    const int threads = T <= 148 ? 512 : 256;                        // few tokens: a token's heads side by side
    if (widest <= 128) launch_pdl(grouped_prep_vec_kernel<16>, dim3(T), dim3(threads), 0, (cudaStream_t)stream, a);
    else launch_pdl(grouped_prep_vec_kernel<32>, dim3(T), dim3(threads), 0, (cudaStream_t)stream, a);
    return cudaGetLastError() == cudaSuccess ? 0 : -4;
  }
  const long long warps = static_cast<long long>(T) * (heads + kv_heads);
  const dim3 grid(static_cast<unsigned>((warps + kGqWarps - 1) / kGqWarps));
  cudaStream_t st = (cudaStream_t)stream;
  if (fp32) launch_pdl(grouped_prep_kernel<float>, grid, dim3(kGqWarps * 32), 0, st, a, vec_in, vec_row);
  else launch_pdl(grouped_prep_kernel<__nv_bfloat16>, grid, dim3(kGqWarps * 32), 0, st, a, vec_in, vec_row);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
