// Grouped-query attention whose heads' scores are mixed before the softmax (ops/talking.py).
//
// A cached row holds the values of all key/value heads (vp columns each), then from k_col on their keys (kp columns each); pages are
// [64][row].  A mixed query has G * kp columns: in the part of key/value head c the sum of talk[h, g] q_g over the heads g that read c.
//
//   talking_prep         one CTA per token, or a few where there are few tokens: biases, weighted RMS norms, rotation, the token's row, mixed queries, gate logits
//   talking_simt         any size and type, fp32 arithmetic throughout: one CTA per (token, head)
#define STK_PDL_CLASS 8
#include "hybrid_block.cuh"
#include "talking_attention.cuh"

namespace stk {

struct TalkPrepArgs {
  const void* proj; long long ldp; int q_off, k_off, v_off, g_off;
  const float* bias;                                   // [H * D | G * D | G * V] or nullptr
  const float* q_norm; const float* k_norm; float eps; // [D] or nullptr
  const float* freq; int pairs;                        // [2][pairs]
  const float* talk;                                   // [H, H]
  const int64_t* positions; const int* tok_req; const int* table; int bt_stride;
  void* cache; int row, k_col, kp, vp;
  int H, G, D, V, T;
  void* q; float* gate;
};

__device__ __forceinline__ void talk_load4(const float* p, float (&v)[4]) {
  const float4 f = *reinterpret_cast<const float4*>(p);
  v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
}
__device__ __forceinline__ void talk_load4(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
}

// HG: heads per key/value head (their queries stay in registers while the heads' mixtures are formed), 0: any number.  grid (T, parts): a
// part forms the mixtures of its share of the heads; the first one also writes the cached row and the gate logits.
// VEC: heads of at most 128 columns in whole aligned groups of four.
template <typename A, int HG, bool VEC>
__global__ void __launch_bounds__(512)
talking_prep_kernel(const TalkPrepArgs a) {
  extern __shared__ __align__(16) float sm[];
  const int D2 = (a.D + 3) & ~3, H4 = (a.H + 3) & ~3;
  float* x = sm;                                       // [H + G][D2]: queries, keys
  float* talk = x + (a.H + a.G) * D2;                  // [heads of this part][H4]
  const int per = (a.H + gridDim.y - 1) / gridDim.y, h0 = blockIdx.y * per, h1 = min(a.H, h0 + per);
  float2* cs = reinterpret_cast<float2*>(talk + per * H4);      // [pairs]
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, KD = a.G * a.kp, warps = blockDim.x >> 5;
  const bool lead = blockIdx.y == 0;
  const int req = a.tok_req[t];
  const long long pos = a.positions[t];
  A* q = reinterpret_cast<A*>(a.q) + t * KD;           // head h: h * T * KD further
  const long long hstep = static_cast<long long>(a.T) * KD;
  const A* p = reinterpret_cast<const A*>(a.proj) + t * a.ldp;
  if (lead && a.gate != nullptr)
    for (int h = threadIdx.x; h < a.H; h += blockDim.x) a.gate[t * a.H + h] = ld_act(p + a.g_off + h);
  if (req < 0 || pos < 0) {
    for (int h = h0; h < h1; ++h)
      for (int i = threadIdx.x; i < KD; i += blockDim.x) st_act(q + h * hstep + i, 0.f);
    return;
  }
  const int page = a.table[static_cast<long long>(req) * a.bt_stride + pos / kTkPage];
  for (int i = threadIdx.x; i < a.pairs; i += blockDim.x) cs[i] = cos_sin_split(pos, a.freq[i], a.freq[a.pairs + i]);
  for (int h = h0 + warp; h < h1; h += warps)
    for (int i = lane; i < a.H; i += 32) talk[(h - h0) * H4 + i] = a.talk[h * a.H + i];
  __syncthreads();
  if (VEC) {
    // four neighbouring columns per lane: norm and rotation in registers
    for (int u0 = warp; u0 < a.H + a.G; u0 += warps) {
      const bool isq = u0 < a.H;
      const A* src = p + (isq ? a.q_off + u0 * a.D : a.k_off + (u0 - a.H) * a.D);
      const float* w = isq ? a.q_norm : a.k_norm;
      const int d = lane * 4;
      float v[4] = {0.f, 0.f, 0.f, 0.f};
      if (d < a.D) {
        talk_load4(src + d, v);
        if (a.bias != nullptr) {
          const float4 b = *reinterpret_cast<const float4*>(a.bias + u0 * a.D + d);
          v[0] += b.x; v[1] += b.y; v[2] += b.z; v[3] += b.w;
        }
      }
      if (w != nullptr) {
        const float s = fmaf(v[0], v[0], fmaf(v[1], v[1], fmaf(v[2], v[2], v[3] * v[3])));
        const float f = 1.f / sqrtf(warp_sum(s) / static_cast<float>(a.D) + a.eps);
        if (d < a.D) {
          const float4 y = *reinterpret_cast<const float4*>(w + d);
          v[0] *= f * y.x; v[1] *= f * y.y; v[2] *= f * y.z; v[3] *= f * y.w;
        }
      }
      if (d >= a.D) continue;
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (lane * 2 + j < a.pairs) {
          const float2 c = cs[lane * 2 + j];
          const float x0 = v[2 * j], x1 = v[2 * j + 1];
          v[2 * j] = x0 * c.x - x1 * c.y;
          v[2 * j + 1] = x1 * c.x + x0 * c.y;
        }
      *reinterpret_cast<float4*>(x + u0 * D2 + d) = make_float4(v[0], v[1], v[2], v[3]);
    }
  } else {
    for (int u0 = warp; u0 < a.H + a.G; u0 += warps) {
      const bool isq = u0 < a.H;
      const A* src = p + (isq ? a.q_off + u0 * a.D : a.k_off + (u0 - a.H) * a.D);
      const float* w = isq ? a.q_norm : a.k_norm;
      float* dst = x + u0 * D2;
      float s = 0.f;
      for (int d = lane; d < D2; d += 32) {
        const float v = d < a.D ? ld_act(src + d) + (a.bias != nullptr ? a.bias[u0 * a.D + d] : 0.f) : 0.f;
        dst[d] = v;
        s = fmaf(v, v, s);
      }
      if (w != nullptr) {
        const float f = 1.f / sqrtf(warp_sum(s) / static_cast<float>(a.D) + a.eps);
        for (int d = lane; d < a.D; d += 32) dst[d] *= f * w[d];
      }
      __syncwarp();
      for (int i = lane; i < a.pairs; i += 32) {
        float2* v = reinterpret_cast<float2*>(dst + 2 * i);
        const float2 c = *v, w2 = cs[i];
        *v = make_float2(c.x * w2.x - c.y * w2.y, c.y * w2.x + c.x * w2.y);
      }
    }
  }
  __syncthreads();
  if (lead && page >= 0) {
    A* row = reinterpret_cast<A*>(a.cache) + (static_cast<long long>(page) * kTkPage + pos % kTkPage) * a.row;
    for (int g = warp; g < a.G; g += warps) {
      const A* v = p + a.v_off + g * a.V;
      const float* b = a.bias != nullptr ? a.bias + (a.H + a.G) * a.D + g * a.V : nullptr;
      for (int d = lane; d < a.vp; d += 32) st_act(row + g * a.vp + d, d < a.V ? ld_act(v + d) + (b != nullptr ? b[d] : 0.f) : 0.f);
      for (int d = lane; d < a.kp; d += 32) st_act(row + a.k_col + g * a.kp + d, d < a.D ? x[(a.H + g) * D2 + d] : 0.f);
    }
  }
  // four columns of the mixtures of every other, fourth, ... head (kp is a multiple of 4)
  const int hg = HG > 0 ? HG : a.H / a.G, quads = a.kp >> 2, items = a.G * quads;
  const int lots = max(1, min(h1 - h0, static_cast<int>(blockDim.x) / items));
  for (int e = threadIdx.x; e < items * lots; e += blockDim.x) {
    const int lot = e / items, i = e - lot * items, c = i / quads, d = (i - c * quads) * 4;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const float* qc = x + c * hg * D2 + d;
    float4 qv[HG > 0 ? HG : 1];
    if (HG > 0) {
#pragma unroll
      for (int g = 0; g < HG; ++g) qv[g] = d < a.D ? *reinterpret_cast<const float4*>(qc + g * D2) : zero;
    }
    for (int h = h0 + lot; h < h1; h += lots) {
      const float* w = talk + (h - h0) * H4 + c * hg;
      float4 s = zero;
      if (HG > 0 && HG % 4 == 0) {
#pragma unroll
        for (int g0 = 0; g0 < HG; g0 += 4) {
          const float4 wv = *reinterpret_cast<const float4*>(w + g0);
          const float wg[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
          for (int g = 0; g < 4; ++g) {
            const float4 y = qv[HG > 0 ? g0 + g : 0];
            s.x = fmaf(wg[g], y.x, s.x); s.y = fmaf(wg[g], y.y, s.y);
            s.z = fmaf(wg[g], y.z, s.z); s.w = fmaf(wg[g], y.w, s.w);
          }
        }
      } else if (HG > 0) {
#pragma unroll
        for (int g = 0; g < HG; ++g) {
          s.x = fmaf(w[g], qv[g].x, s.x); s.y = fmaf(w[g], qv[g].y, s.y);
          s.z = fmaf(w[g], qv[g].z, s.z); s.w = fmaf(w[g], qv[g].w, s.w);
        }
      } else if (d < a.D) {
        for (int g = 0; g < hg; ++g) {
          const float4 y = *reinterpret_cast<const float4*>(qc + g * D2);
          s.x = fmaf(w[g], y.x, s.x); s.y = fmaf(w[g], y.y, s.y);
          s.z = fmaf(w[g], y.z, s.z); s.w = fmaf(w[g], y.w, s.w);
        }
      }
      A* to = q + h * hstep + c * a.kp + d;
      if constexpr (sizeof(A) == 2) {
        __align__(8) const __nv_bfloat162 b[2] = {__floats2bfloat162_rn(s.x, s.y), __floats2bfloat162_rn(s.z, s.w)};
        *reinterpret_cast<uint2*>(to) = *reinterpret_cast<const uint2*>(b);
      } else {
        *reinterpret_cast<float4*>(to) = s;
      }
    }
  }
}

// ---- any size, fp32 arithmetic ------------------------------------------------------------------
constexpr int kTkKeys = 512;

template <typename A>
__global__ void __launch_bounds__(128)
talking_simt_kernel(const TalkArgs a, const int* __restrict__ first_pos, const int* __restrict__ last_pos, int max_span) {
  extern __shared__ __align__(16) float q[];           // [G * kp]
  __shared__ float sc[kTkKeys];
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x, h = blockIdx.y, KD = a.G * a.kp, vc = h / (a.H / a.G) * a.vp;
  const int req = a.tok_req[t];
  const long long pos = a.positions[t];
  A* out = reinterpret_cast<A*>(a.out) + t * a.ldo;
  if (req >= 0 && pos >= 0 && last_pos[t] - first_pos[t] + 1 > max_span) return;
  if (h == a.H - 1)
    for (int d = a.H * a.V + threadIdx.x; d < a.out_cols; d += blockDim.x) st_act(out + d, 0.f);
  out += h * a.V;
  if (req < 0 || pos < 0) {
    for (int d = threadIdx.x; d < a.V; d += blockDim.x) st_act(out + d, 0.f);
    return;
  }
  const A* qg = reinterpret_cast<const A*>(a.q) + (static_cast<long long>(h) * a.T + t) * KD;
  for (int d = threadIdx.x; d < KD; d += blockDim.x) q[d] = ld_act(qg + d);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long lo = talk_first(a, pos);
  const int* bt = a.table + static_cast<long long>(req) * a.bt_stride;
  const A* cache = reinterpret_cast<const A*>(a.cache);
  auto row_of = [&](long long p) {
    const int page = bt[p / kTkPage];
    return cache + (static_cast<long long>(page < 0 ? 0 : page) * kTkPage + p % kTkPage) * a.row;
  };
  float m = a.sink != nullptr ? a.sink[h] : -INFINITY, l = a.sink != nullptr ? 1.f : 0.f, acc[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) acc[i] = 0.f;
  for (long long k0 = lo; k0 <= pos; k0 += kTkKeys) {
    const int n = static_cast<int>(pos + 1 - k0 < kTkKeys ? pos + 1 - k0 : kTkKeys);
    float mx = -INFINITY;
    for (int j = warp; j < n; j += 4) {
      const A* r = row_of(k0 + j) + a.k_col;
      float s = 0.f;
      for (int d = lane; d < KD; d += 32) s = fmaf(q[d], ld_act(r + d), s);
      s = warp_sum(s) * a.scale;
      if (lane == 0) sc[j] = s;
      mx = fmaxf(mx, s);
    }
    const float m_new = fmaxf(m, block_max(mx, red));
    float sum = 0.f;
    for (int j = threadIdx.x; j < n; j += blockDim.x) {
      const float p = expf(sc[j] - m_new);
      sc[j] = p;
      sum += p;
    }
    const float f = expf(m - m_new);
    l = l * f + block_sum(sum, red);
    m = m_new;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[i] *= f;
    for (int j = 0; j < n; ++j) {
      const A* r = row_of(k0 + j) + vc;
      const float p = sc[j];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int d = threadIdx.x + i * 128;
        if (d < a.V) acc[i] = fmaf(p, ld_act(r + d), acc[i]);
      }
    }
    __syncthreads();
  }
  const float g = talk_gate(a, t, h) / l;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int d = threadIdx.x + i * 128;
    if (d < a.V) st_act(out + d, acc[i] * g);
  }
}

template <typename A>
static int launch_talk_prep(const TalkPrepArgs& a, int T, cudaStream_t st) {
  const int parts = T >= 148 ? 1 : min((a.H + 3) / 4, 8), per = (a.H + parts - 1) / parts, threads = T >= 148 ? 256 : 512;
  const size_t smem = (static_cast<size_t>(a.H + a.G) * ((a.D + 3) & ~3) + per * ((a.H + 3) & ~3) + 2 * a.pairs) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  const uintptr_t at = reinterpret_cast<uintptr_t>(a.proj);
  const bool vec = a.D % 4 == 0 && a.D <= 128 && a.ldp % 4 == 0 && (a.q_off | a.k_off) % 4 == 0 && (at & 15) == 0 &&
                   ((reinterpret_cast<uintptr_t>(a.bias) | reinterpret_cast<uintptr_t>(a.q_norm) | reinterpret_cast<uintptr_t>(a.k_norm)) & 15) == 0;
#define STK_TALK_PREP_AS(HG, VEC)                                                                                               \
  {                                                                                                                             \
    if (smem > 40 * 1024 && cudaFuncSetAttribute(talking_prep_kernel<A, HG, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize,  \
                                                 200 * 1024) != cudaSuccess)                                                    \
      return -3;                                                                                                                \
    launch_pdl(talking_prep_kernel<A, HG, VEC>, dim3(T, parts), dim3(threads), smem, st, a);                                    \
  }
#define STK_TALK_PREP(HG)                 \
  if (vec) STK_TALK_PREP_AS(HG, true)     \
  else STK_TALK_PREP_AS(HG, false)
  switch (a.H / a.G) {
    case 1: STK_TALK_PREP(1) break;
    case 2: STK_TALK_PREP(2) break;
    case 4: STK_TALK_PREP(4) break;
    case 8: STK_TALK_PREP(8) break;
    default: STK_TALK_PREP(0) break;
  }
#undef STK_TALK_PREP
#undef STK_TALK_PREP_AS
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

}  // namespace stk

using namespace stk;

// q: [heads, T, kv_heads * kp] in the type of proj, 16-byte aligned; gate [T, heads] fp32 or null (no gate).
STK_API int stk_talking_prep(const void* proj, long long ldp, int q_off, int k_off, int v_off, int g_off, const float* bias,
                             const float* q_norm, const float* k_norm, float eps, const float* freq, int pairs, const float* talk,
                             const int64_t* positions, const int* tok_req, const int* table, int bt_stride, void* cache, int row, int k_col,
                             int kp, int vp, int heads, int kv_heads, int dim, int vdim, void* q, float* gate, int fp32, int T,
                             void* stream) {
  if (T <= 0) return 0;
  if (heads < 1 || kv_heads < 1 || heads % kv_heads || dim < 1 || vdim < 1 || kp < dim || (kp & 15) || vp < vdim || k_col != kv_heads * vp ||
      row < k_col + kv_heads * kp || pairs < 0 || 2 * pairs > dim || (q_norm == nullptr) != (k_norm == nullptr) || (reinterpret_cast<uintptr_t>(q) & 15))
    return -1;
  TalkPrepArgs a;
  a.proj = proj; a.ldp = ldp; a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.g_off = g_off;
  a.bias = bias; a.q_norm = q_norm; a.k_norm = k_norm; a.eps = eps; a.freq = freq; a.pairs = pairs; a.talk = talk;
  a.positions = positions; a.tok_req = tok_req; a.table = table; a.bt_stride = bt_stride;
  a.cache = cache; a.row = row; a.k_col = k_col; a.kp = kp; a.vp = vp;
  a.H = heads; a.G = kv_heads; a.D = dim; a.V = vdim; a.T = T; a.q = q; a.gate = gate;
  return fp32 ? launch_talk_prep<float>(a, T, (cudaStream_t)stream) : launch_talk_prep<__nv_bfloat16>(a, T, (cudaStream_t)stream);
}

// Spans of at most max_span tokens.
STK_API int stk_talking_simt(const void* q, const float* gate, const float* sink, const int64_t* positions, const int* tok_req,
                             const int* table, int bt_stride, const void* cache, int row, int k_col, int kp, int vp, int heads, int kv_heads,
                             int vdim, int chunk, float scale, void* out, long long ldo, int out_cols, int fp32, const int* first_pos,
                             const int* last_pos, int max_span, int T, void* stream) {
  if (T <= 0) return 0;
  const TalkArgs a = {q, T, gate, sink, positions, tok_req, table, bt_stride, cache, row, k_col, kp, vp, heads, kv_heads, vdim, chunk,
                      scale, out, ldo, out_cols};
  const size_t smem = static_cast<size_t>(kv_heads) * kp * sizeof(float);
  if (!talk_ok(a) || vdim > 1024 || heads > 65535 || smem > 200 * 1024) return -1;
  cudaStream_t st = (cudaStream_t)stream;
  if (smem > 40 * 1024 &&
      (cudaFuncSetAttribute(talking_simt_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess ||
       cudaFuncSetAttribute(talking_simt_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess))
    return -3;
  if (fp32) launch_pdl(talking_simt_kernel<float>, dim3(T, heads), dim3(128), smem, st, a, first_pos, last_pos, max_span);
  else launch_pdl(talking_simt_kernel<__nv_bfloat16>, dim3(T, heads), dim3(128), smem, st, a, first_pos, last_pos, max_span);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
