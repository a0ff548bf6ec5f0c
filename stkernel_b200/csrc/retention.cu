// Retention: a linear recurrence (linear_scan.cuh) with a fixed decay per head over rotated queries and keys; every head's read-out
// is divided by its root mean square and multiplied with silu of a gate.
//
//   retention_scan       decode rows, short spans, float32: rotation in fp32 on the way into the recurrence
//   rotate_qk            long spans: rotated queries and scaled, rotated keys as bf16 pairs for the chunked form
//   retention_finish     head norm (weighted, if there is a weight), gate, factor; time mixing ends with it as well
#define STK_PDL_CLASS 16
#include "linear_scan.cuh"

namespace stk {

struct RotArgs {
  const void* proj; long long ldp; int q_off, k_off;
  const float* freq; int pairs;                   // [2][pairs]: dimension i turns with i + pairs
  float k_scale;
};

// Element d of a head after its rotation at position pos.
template <typename A>
__device__ __forceinline__ float rotated(const RotArgs& r, const A* x, int d, long long pos) {
  const float v = ld_act(x + d);
  if (d >= 2 * r.pairs) return v;
  const int i = d < r.pairs ? d : d - r.pairs;
  const float2 w = cos_sin_split(pos, r.freq[i], r.freq[r.pairs + i]);
  return d < r.pairs ? v * w.x - ld_act(x + d + r.pairs) * w.y : v * w.x + ld_act(x + d - r.pairs) * w.y;
}

template <typename A>
struct RetentionFront {
  static constexpr bool kPerChannel = false;
  RotArgs r;
  int v_off, D, V;
  const float* decay;                             // [2][H]: the decays and what their rounding left over
  int H;
  __device__ __forceinline__ float skip(int) const { return 0.f; }
  __device__ __forceinline__ float value(long long t, int h, int col) const {
    return ld_act(reinterpret_cast<const A*>(r.proj) + t * r.ldp + v_off + h * V + col);
  }
  __device__ __forceinline__ float2 fill(long long t, long long pos, int h, float* q, float* k) const {
    const A* p = reinterpret_cast<const A*>(r.proj) + t * r.ldp;
    for (int e = threadIdx.x; e < 2 * D; e += kScanThreads) {
      if (e < D) q[e] = rotated(r, p + r.q_off + h * D, e, pos);
      else k[e - D] = rotated(r, p + r.k_off + h * D, e - D, pos) * r.k_scale;
    }
    return make_float2(decay[h], decay[H + h]);
  }
};

// Eight fp32 values as bf16 high parts and remainders, `n` elements apart.
__device__ __forceinline__ void store_pair8(__nv_bfloat16* dst, int n, const float (&y)[8]) {
  uint4 hi, lo;
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(y[2 * j], y[2 * j + 1]);
    const float2 f = __bfloat1622float2(h);
    reinterpret_cast<__nv_bfloat162*>(&hi)[j] = h;
    reinterpret_cast<__nv_bfloat162*>(&lo)[j] = __floats2bfloat162_rn(y[2 * j] - f.x, y[2 * j + 1] - f.y);
  }
  *reinterpret_cast<uint4*>(dst) = hi;
  *reinterpret_cast<uint4*>(dst + n) = lo;
}
__device__ __forceinline__ void load8(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 u = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&v)[j]);
    f[2 * j] = u.x;
    f[2 * j + 1] = u.y;
  }
}

// out [T][q high | q remainder | k high | k remainder][H * D8], zeros behind each head's D columns.  One CTA per token; the cos and
// sin of its position are formed once for all heads.  vec: heads, rotated pairs and rows in whole groups of eight.
__global__ void __launch_bounds__(256)
rotate_qk_kernel(const RotArgs r, const int64_t* __restrict__ positions, __nv_bfloat16* __restrict__ out, int H, int D, int D8, int vec) {
  extern __shared__ float2 cs[];
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const long long pos = positions[t] < 0 ? 0 : positions[t];
  for (int i = threadIdx.x; i < r.pairs; i += blockDim.x) cs[i] = cos_sin_split(pos, r.freq[i], r.freq[r.pairs + i]);
  __syncthreads();
  const __nv_bfloat16* p = reinterpret_cast<const __nv_bfloat16*>(r.proj) + t * r.ldp;
  const int n = H * D8;
  __nv_bfloat16* o = out + t * 4 * n;
  if (vec) {
    const int turned = r.pairs >> 3, items = turned + ((D - 2 * r.pairs) >> 3);      // per head: pairs of groups, then plain groups
    for (int e = threadIdx.x; e < 2 * H * items; e += blockDim.x) {
      const int u = e / items, i = e - u * items, isk = u >= H ? 1 : 0, h = u - isk * H;
      const __nv_bfloat16* x = p + (isk ? r.k_off : r.q_off) + h * D;
      __nv_bfloat16* dst = o + isk * 2 * n + h * D8;
      const float f = isk ? r.k_scale : 1.f;
      float a[8], b[8], y[8], z[8];
      if (i < turned) {
        load8(x + i * 8, a);
        load8(x + r.pairs + i * 8, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const float2 w = cs[i * 8 + j];
          y[j] = (a[j] * w.x - b[j] * w.y) * f;
          z[j] = (b[j] * w.x + a[j] * w.y) * f;
        }
        store_pair8(dst + i * 8, n, y);
        store_pair8(dst + r.pairs + i * 8, n, z);
      } else {
        const int d = 2 * r.pairs + (i - turned) * 8;
        load8(x + d, a);
#pragma unroll
        for (int j = 0; j < 8; ++j) y[j] = a[j] * f;
        store_pair8(dst + d, n, y);
      }
    }
    return;
  }
  for (int e = threadIdx.x; e < n; e += blockDim.x) {               // two columns, e / (D8 / 2) the (q or k, head)
    const int half = D8 / 2, u = e / half, d0 = (e - u * half) * 2, isk = u >= H ? 1 : 0, h = u - isk * H;
    const __nv_bfloat16* x = p + (isk ? r.k_off : r.q_off) + h * D;
    float y[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int d = d0 + j;
      float f = 0.f;
      if (d < D) {
        f = bf16_to_f(x[d]);
        if (d < 2 * r.pairs) {
          const float2 w = cs[d < r.pairs ? d : d - r.pairs];
          f = d < r.pairs ? f * w.x - bf16_to_f(x[d + r.pairs]) * w.y : f * w.x + bf16_to_f(x[d - r.pairs]) * w.y;
        }
        if (isk) f *= r.k_scale;
      }
      y[j] = f;
    }
    const __nv_bfloat162 hi = __floats2bfloat162_rn(y[0], y[1]);
    const float2 hf = __bfloat1622float2(hi);
    __nv_bfloat16* dst = o + isk * 2 * n + h * D8 + d0;
    *reinterpret_cast<__nv_bfloat162*>(dst) = hi;
    *reinterpret_cast<__nv_bfloat162*>(dst + n) = __floats2bfloat162_rn(y[0] - hf.x, y[1] - hf.y);
  }
}

// out[t, col + h * V + c] = o / rms(o over the head) * weight * silu(g) * scale (weight null: 1): one warp per (token, head).  Zeros into the columns left .. col
// and behind the last head.  NV > 0: bf16 heads of at most 4 * LPH * NV columns in whole groups of
// four, which stay in registers, LPH lanes per (token, head).
template <typename A, int NV, int LPH>
__global__ void __launch_bounds__(256)
retention_finish_kernel(const float* __restrict__ o, float eps, const float* __restrict__ weight, const int* __restrict__ tok_req, const int64_t* __restrict__ positions,
                        const A* __restrict__ proj, long long ldp, int g_off, float scale, A* __restrict__ out, long long ldo, int left,
                        int col, int cols, int H, int V, int T) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & (LPH - 1);
  const long long th = blockIdx.x * (256ll / LPH) + threadIdx.x / LPH;
  if (th >= static_cast<long long>(T) * H) return;
  const unsigned mates = LPH == 32 ? 0xffffffffu : 0xffffu << (threadIdx.x & 16);
  auto head_sum = [&](float v) {
#pragma unroll
    for (int o = LPH / 2; o > 0; o >>= 1) v += __shfl_xor_sync(mates, v, o);
    return v;
  };
  const long long t = th / H;
  const int h = static_cast<int>(th - t * H);
  A* to = out + t * ldo;
  const float* x = o + th * V;
  const A* g = proj + t * ldp + g_off + h * V;
  float4 v[NV > 0 ? NV : 1];
  uint2 gu[NV > 0 ? NV : 1];
  if (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * LPH + lane) * 4;
      v[i] = c < V ? *reinterpret_cast<const float4*>(x + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      gu[i] = c < V ? *reinterpret_cast<const uint2*>(g + c) : make_uint2(0, 0);
    }
  }
  if (h == 0)
    for (int c = left + lane; c < col; c += LPH) st_act(to + c, 0.f);
  if (h == H - 1)
    for (int c = col + H * V + lane; c < cols; c += LPH) st_act(to + c, 0.f);
  to += col + h * V;
  if (tok_req[t] < 0 || positions[t] < 0) {
    for (int c = lane; c < V; c += LPH) st_act(to + c, 0.f);
    return;
  }
  float ss = 0.f;
  if (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) ss = fmaf(v[i].x, v[i].x, fmaf(v[i].y, v[i].y, fmaf(v[i].z, v[i].z, fmaf(v[i].w, v[i].w, ss))));
    const float r = scale / sqrtf(head_sum(ss) / static_cast<float>(V) + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * LPH + lane) * 4;
      if (c >= V) continue;
      const float2 g0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gu[i].x));
      const float2 g1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gu[i].y));
      if (weight != nullptr) {
        const float4 w = *reinterpret_cast<const float4*>(weight + h * V + c);
        v[i].x *= w.x; v[i].y *= w.y; v[i].z *= w.z; v[i].w *= w.w;
      }
      uint2 pk;
      *reinterpret_cast<__nv_bfloat162*>(&pk.x) = __floats2bfloat162_rn(v[i].x * r * silu_bf16(g0.x), v[i].y * r * silu_bf16(g0.y));
      *reinterpret_cast<__nv_bfloat162*>(&pk.y) = __floats2bfloat162_rn(v[i].z * r * silu_bf16(g1.x), v[i].w * r * silu_bf16(g1.y));
      *reinterpret_cast<uint2*>(to + c) = pk;
    }
    return;
  }
  for (int c = lane; c < V; c += LPH) ss = fmaf(x[c], x[c], ss);
  const float r = scale / sqrtf(head_sum(ss) / static_cast<float>(V) + eps);
  for (int c = lane; c < V; c += LPH) {
    const float z = ld_act(g + c);
    st_act(to + c, x[c] * r * (weight != nullptr ? weight[h * V + c] : 1.f) * z / (1.f + expf(-z)));
  }
}

}  // namespace stk

using namespace stk;

// Spans of min_span .. max_span tokens, token by token.
STK_API int stk_retention_scan(const void* proj, long long ldp, int q_off, int k_off, int v_off, const float* freq, int pairs,
                               float k_scale, const float* decay, const int* query_start, const int* req_rows, const int* start_pos,
                               int n_req, float* S, float* o, int heads, int dim, int vdim, int fp32, int min_span, int max_span, int T,
                               void* stream) {
  if (T <= 0) return 0;
  if (pairs < 0 || 2 * pairs > dim) return -1;
  const ScanArgs a{query_start, req_rows, start_pos, n_req, S, o, heads, dim, vdim};
  const RotArgs r{proj, ldp, q_off, k_off, freq, pairs, k_scale};
  if (fp32) return launch_scan(RetentionFront<float>{r, v_off, dim, vdim, decay, heads}, a, min_span, max_span, (cudaStream_t)stream);
  return launch_scan(RetentionFront<__nv_bfloat16>{r, v_off, dim, vdim, decay, heads}, a, min_span, max_span, (cudaStream_t)stream);
}

// out [T, 4, heads * d8] bf16: see rotate_qk_kernel.
STK_API int stk_rotate_qk(const void* proj, long long ldp, int q_off, int k_off, const float* freq, int pairs, float k_scale,
                          const int64_t* positions, void* out, int heads, int dim, int d8, int T, void* stream) {
  if (T <= 0) return 0;
  if (pairs < 0 || 2 * pairs > dim || d8 < dim || d8 % 8) return -1;
  const RotArgs r{proj, ldp, q_off, k_off, freq, pairs, k_scale};
  const int vec = pairs % 8 == 0 && dim % 8 == 0 && ldp % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 &&
                  ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  launch_pdl(rotate_qk_kernel, dim3(T), dim3(256), static_cast<size_t>(pairs) * sizeof(float2), (cudaStream_t)stream, r, positions,
             (__nv_bfloat16*)out, heads, dim, d8, vec);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_retention_finish(const float* o, float eps, const float* weight, const int* tok_req, const int64_t* positions, const void* proj, long long ldp,
                                 int g_off, float scale, void* out, long long ldo, int left, int col, int cols, int fp32, int heads,
                                 int vdim, int T, void* stream) {
  if (T <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  const bool vec = !fp32 && vdim <= 512 && ((vdim | g_off | col) & 3) == 0 && (reinterpret_cast<uintptr_t>(weight) & 15) == 0 && ((ldp | ldo) & 3) == 0 &&
                   ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(out)) & 7) == 0;
#define STK_FINISH(A, NV, LPH)                                                                                                     \
  launch_pdl(retention_finish_kernel<A, NV, LPH>, dim3(static_cast<unsigned>((static_cast<long long>(T) * heads + 256 / LPH - 1) / (256 / LPH))), dim3(256), 0, st, o, eps, weight, tok_req, positions, (const A*)proj, ldp, g_off, scale, (A*)out, \
             ldo, left, col, cols, heads, vdim, T)
  if (fp32) STK_FINISH(float, 0, 32);
  else if (!vec) STK_FINISH(__nv_bfloat16, 0, 32);
  else if (vdim <= 64) STK_FINISH(__nv_bfloat16, 1, 16);
  else if (vdim <= 128) STK_FINISH(__nv_bfloat16, 1, 32);
  else if (vdim <= 256) STK_FINISH(__nv_bfloat16, 2, 32);
  else STK_FINISH(__nv_bfloat16, 4, 32);
#undef STK_FINISH
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
