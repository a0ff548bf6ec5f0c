// Mamba-2: a linear recurrence (linear_scan.cuh) with k = dt B, q = C, v = x and log decay -exp(A) dt, whose operands x, B and C come
// through a short causal convolution per channel and silu.
//
//   mamba2_conv        convolved operands in the compute type, step sizes and log decays
//   mamba2_scan        decode rows, short spans, float32 (long spans: linear_scan.cu)
//   mamba2_finish      gate silu(z), RMS norm in equal parts, and the last convolution inputs of every span into its request's ring
//
// Convolution inputs before a span come from ring [rows][taps - 1][channels] (position p at p mod (taps - 1)), those before
// position 0 are zero.  The ring is written after everything that reads it has run.
#define STK_PDL_CLASS 16
#include "linear_scan.cuh"

namespace stk {

struct ConvArgs {
  const void* proj; long long ldp; int x_off, dt_off;
  const float* taps; const float* bias; int n;    // [n][channels], current token last; [channels]
  const void* ring;
  const float* dt_bias; const float* neg_a;       // [H]
  int channels;
};

__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

template <typename A>
struct Mamba2Front {
  static constexpr bool kPerChannel = false;
  const A* xbc; long long ld;                     // [T, ld]: x | B | C, convolved
  const float* steps;                             // [2][H][T]: log decays, step sizes
  int N, V, inner, groups, hpg, H, T;
  const float* skips;
  __device__ __forceinline__ float skip(int h) const { return skips[h]; }
  __device__ __forceinline__ float value(long long t, int h, int col) const { return ld_act(xbc + t * ld + h * V + col); }
  __device__ __forceinline__ float2 fill(long long t, long long, int h, float* q, float* k) const {
    const long long at = static_cast<long long>(h) * T + t;
    const float lg = steps[at], dt = steps[static_cast<long long>(H) * T + at];
    const A* p = xbc + t * ld + inner + h / hpg * N;
    for (int e = threadIdx.x; e < 2 * N; e += kScanThreads) {
      if (e < N) k[e] = ld_act(p + e) * dt;
      else q[e - N] = ld_act(p + groups * N + e - N);
    }
    // slow decays as 1 and the (small) difference from it: a rounded factor close to 1 would be off in the same direction for long
    return lg > -0.25f ? make_float2(1.f, expm1f(lg)) : make_float2(expf(lg), 0.f);
  }
};

constexpr int kConvTok = 32, kConvBatch = 4, kConvCh = 4, kConvThreads = 256;

// Four channels x TOK tokens per thread.  NT > 0 taps: the inputs of tokens that follow one another in one span slide through
// registers, a batch of kConvBatch in flight while the one before is summed; otherwise (spans that meet inside the group, many
// taps, unaligned rows) every tap is read where it is used.  The grid's last column of blocks forms the step sizes.
template <typename A, int NT, int TOK>
__global__ void __launch_bounds__(kConvThreads, TOK > 1 && NT > 0 ? 4 : 1)
mamba2_conv_kernel(const ConvArgs a, const int64_t* __restrict__ positions, const int* __restrict__ tok_req,
                   const int* __restrict__ first_pos, A* __restrict__ out, long long ldo, float* __restrict__ steps, int H, int T,
                   int vec) {
  pdl_wait();
  pdl_trigger();
  const A* proj = reinterpret_cast<const A*>(a.proj);
  const int t0 = blockIdx.y * TOK, t1 = min(T, t0 + TOK);
  if (blockIdx.x == gridDim.x - 1) {
    // steps [0][H][T]: log decays, [1][H][T]: step sizes
    for (int e = threadIdx.x; e < TOK * H; e += kConvThreads) {
      const int h = e / TOK, t = t0 + e % TOK;
      if (t >= T) continue;
      const float dt = softplus_f(ld_act(proj + t * a.ldp + a.dt_off + h) + a.dt_bias[h]);
      steps[static_cast<long long>(h) * T + t] = dt * a.neg_a[h];
      steps[(static_cast<long long>(H) + h) * T + t] = dt;
    }
    return;
  }
  const int ch = (blockIdx.x * kConvThreads + threadIdx.x) * kConvCh;
  if (ch >= ldo) return;
  const int nc = min(kConvCh, a.channels - ch), keep = a.n - 1;
  const A* x = proj + a.x_off + ch;
  const A* ring = reinterpret_cast<const A*>(a.ring) + ch;
  auto fetch = [&](const A* src, float (&f)[kConvCh]) {
    if (sizeof(A) == 2 && vec) {
      uint2 v = make_uint2(0, 0);
      if (src != nullptr) v = *reinterpret_cast<const uint2*>(src);
#pragma unroll
      for (int c = 0; c < kConvCh / 2; ++c) {
        const float2 u = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&v)[c]);
        f[2 * c] = u.x;
        f[2 * c + 1] = u.y;
      }
    } else {
#pragma unroll
      for (int c = 0; c < kConvCh; ++c) f[c] = src != nullptr && c < nc ? ld_act(src + c) : 0.f;
    }
  };
  auto coeff = [&](const float* src, float (&f)[kConvCh]) {
    if (vec) {
      const float4 u = *reinterpret_cast<const float4*>(src);
      f[0] = u.x; f[1] = u.y; f[2] = u.z; f[3] = u.w;
    } else {
#pragma unroll
      for (int c = 0; c < kConvCh; ++c) f[c] = c < nc ? src[c] : 0.f;
    }
  };
  // where the input j tokens before token t is: its own span's row, the ring, or nowhere (zero)
  auto where = [&](int t, int j, int req, long long pos, int first) -> const A* {
    if (pos - j >= first) return x + (t - j) * a.ldp;
    if (pos >= j) return ring + (static_cast<long long>(req) * keep + (pos - j) % keep) * a.channels;
    return nullptr;
  };
  auto put = [&](int t, const float (&s)[kConvCh]) {
    if (sizeof(A) == 2) {
      // behind the last channel the sums are zero, and so is silu
      __align__(8) __nv_bfloat162 b[kConvCh / 2];
#pragma unroll
      for (int c = 0; c < kConvCh / 2; ++c) {
        const float y = s[2 * c], z = s[2 * c + 1];
        b[c] = __floats2bfloat162_rn(silu_bf16(y), silu_bf16(z));
      }
      *reinterpret_cast<uint2*>(out + t * ldo + ch) = *reinterpret_cast<const uint2*>(b);
    } else {
#pragma unroll
      for (int c = 0; c < kConvCh; ++c) st_act(out + t * ldo + ch + c, c < nc ? silu_f(s[c]) : 0.f);
    }
  };
  const int req0 = tok_req[t0], first0 = first_pos[t0];
  const long long pos0 = positions[t0];
  float bias[kConvCh];
  coeff(a.bias + ch, bias);
  if (NT > 0 && vec && req0 >= 0 && pos0 >= 0 && tok_req[t1 - 1] == req0 && positions[t1 - 1] == pos0 + (t1 - 1 - t0)) {
    constexpr int kN = NT > 0 ? NT : 1, kB = TOK < kConvBatch ? TOK : kConvBatch;
    float w[kN][kConvCh];
#pragma unroll
    for (int j = 0; j < kN; ++j) coeff(a.taps + (a.n - 1 - j) * a.channels + ch, w[j]);
    float in[kB + kN - 1][kConvCh];                       // inputs of the kN - 1 tokens before a batch, then the batch's
#pragma unroll
    for (int i = 0; i < kN - 1; ++i) fetch(where(t0, kN - 1 - i, req0, pos0, first0), in[kB + i]);
    uint2 ahead[kB];
    auto request = [&](int b0) {
#pragma unroll
      for (int i = 0; i < kB; ++i)
        ahead[i] = b0 + i < t1 ? *reinterpret_cast<const uint2*>(x + (b0 + i) * a.ldp) : make_uint2(0, 0);
    };
    request(t0);
    for (int b0 = t0; b0 < t1; b0 += kB) {
#pragma unroll
      for (int i = 0; i < kN - 1; ++i)
#pragma unroll
        for (int c = 0; c < kConvCh; ++c) in[i][c] = in[kB + i][c];
#pragma unroll
      for (int i = 0; i < kB; ++i) {
        const float2 u = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&ahead[i].x));
        const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&ahead[i].y));
        float (&f)[kConvCh] = in[kN - 1 + i];
        f[0] = u.x; f[1] = u.y; f[2] = v.x; f[3] = v.y;
      }
      if (b0 + kB < t1) request(b0 + kB);
#pragma unroll
      for (int i = 0; i < kB; ++i) {
        if (b0 + i < t1) {
          float s[kConvCh];
#pragma unroll
          for (int c = 0; c < kConvCh; ++c) {
            s[c] = bias[c];
#pragma unroll
            for (int j = 0; j < kN; ++j) s[c] = fmaf(w[j][c], in[i + kN - 1 - j][c], s[c]);
          }
          put(b0 + i, s);
        }
      }
    }
    return;
  }
  for (int t = t0; t < t1; ++t) {
    const int req = tok_req[t], first = first_pos[t];
    const long long pos = positions[t];
    float s[kConvCh];
#pragma unroll
    for (int c = 0; c < kConvCh; ++c) s[c] = bias[c];
    if (req >= 0 && pos >= 0) {
#pragma unroll 4
      for (int j = 0; j < a.n; ++j) {
        float f[kConvCh], w[kConvCh];
        fetch(where(t, j, req, pos, first), f);
        coeff(a.taps + (a.n - 1 - j) * a.channels + ch, w);
#pragma unroll
        for (int c = 0; c < kConvCh; ++c) s[c] = fmaf(w[c], f[c], s[c]);
      }
    }
    put(t, s);
  }
}

// Convolution inputs of one of a span's last tokens, into its request's ring: this caller's share (part of parts, `threads` wide).
template <typename A>
__device__ __forceinline__ void keep_inputs(const A* x, A* ring, int req, long long pos, int last, int keep, int channels, int part,
                                            int parts, int thread, int threads) {
  if (keep <= 0 || pos <= last - keep) return;
  A* dst = ring + (static_cast<long long>(req) * keep + pos % keep) * channels;
  constexpr int kVec = 16 / sizeof(A);
  if (channels % kVec == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(dst)) & 15) == 0) {
    for (int c = part * threads + thread; c < channels / kVec; c += parts * threads)
      reinterpret_cast<uint4*>(dst)[c] = reinterpret_cast<const uint4*>(x)[c];
    return;
  }
  for (int c = part * threads + thread; c < channels; c += parts * threads) dst[c] = x[c];
}

// One warp per (token, norm part) of at most 128 * NV columns, which stay in registers.
template <int NV>
__global__ void __launch_bounds__(256)
mamba2_finish_warp_kernel(const float* __restrict__ o, const __nv_bfloat16* __restrict__ proj, long long ldp, int z_off, int x_off,
                          int channels, const float* __restrict__ w, float eps, const int* __restrict__ tok_req,
                          const int64_t* __restrict__ positions, const int* __restrict__ last_pos, __nv_bfloat16* __restrict__ ring,
                          int taps, __nv_bfloat16* __restrict__ out, long long ldo, int cols, int inner, int part, int parts, int T) {
  pdl_wait();
  pdl_trigger();
  const int lane = threadIdx.x & 31;
  const long long u = blockIdx.x * 8ll + (threadIdx.x >> 5), t = u / parts;
  if (t >= T) return;
  const int g = static_cast<int>(u - t * parts), c0 = g * part, req = tok_req[t];
  const long long pos = positions[t];
  __nv_bfloat16* to = out + t * ldo;
  if (g == parts - 1)
    for (int c = inner + lane; c < cols; c += 32) to[c] = __float2bfloat16(0.f);
  if (req < 0 || pos < 0) {
    for (int c = lane; c < part; c += 32) to[c0 + c] = __float2bfloat16(0.f);
    return;
  }
  const __nv_bfloat16* p = proj + t * ldp;
  const float4* x = reinterpret_cast<const float4*>(o + t * inner + c0);
  const uint2* z = reinterpret_cast<const uint2*>(p + z_off + c0);
  float4 y[NV];
  uint2 zu[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = i * 32 + lane;
    const bool ok = c * 4 < part;
    y[i] = ok ? x[c] : make_float4(0.f, 0.f, 0.f, 0.f);
    zu[i] = ok ? z[c] : make_uint2(0, 0);
  }
  keep_inputs(p + x_off, ring, req, pos, last_pos[t], taps - 1, channels, g, parts, lane, 32);
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const float2 z0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&zu[i].x));
    const float2 z1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&zu[i].y));
    y[i].x *= silu_bf16(z0.x);
    y[i].y *= silu_bf16(z0.y);
    y[i].z *= silu_bf16(z1.x);
    y[i].w *= silu_bf16(z1.y);
    ss = fmaf(y[i].x, y[i].x, fmaf(y[i].y, y[i].y, fmaf(y[i].z, y[i].z, fmaf(y[i].w, y[i].w, ss))));
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(part) + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = i * 32 + lane;
    if (c * 4 >= part) continue;
    const float4 f = reinterpret_cast<const float4*>(w + c0)[c];
    uint2 pk;
    *reinterpret_cast<__nv_bfloat162*>(&pk.x) = __floats2bfloat162_rn(y[i].x * r * f.x, y[i].y * r * f.y);
    *reinterpret_cast<__nv_bfloat162*>(&pk.y) = __floats2bfloat162_rn(y[i].z * r * f.z, y[i].w * r * f.w);
    reinterpret_cast<uint2*>(to + c0)[c] = pk;
  }
}

// One CTA per (token, norm part).
template <typename A>
__global__ void __launch_bounds__(256)
mamba2_finish_kernel(const float* __restrict__ o, const A* __restrict__ proj, long long ldp, int z_off, int x_off, int channels,
                     const float* __restrict__ w, float eps, const int* __restrict__ tok_req, const int64_t* __restrict__ positions,
                     const int* __restrict__ last_pos, A* __restrict__ ring, int taps, A* __restrict__ out, long long ldo, int cols,
                     int inner, int part) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const int c0 = blockIdx.y * part, req = tok_req[t];
  const long long pos = positions[t];
  A* to = out + t * ldo;
  if (blockIdx.y == gridDim.y - 1)
    for (int c = inner + threadIdx.x; c < cols; c += blockDim.x) st_act(to + c, 0.f);
  if (req < 0 || pos < 0) {
    for (int c = threadIdx.x; c < part; c += blockDim.x) st_act(to + c0 + c, 0.f);
    return;
  }
  const A* p = proj + t * ldp;
  keep_inputs(p + x_off, ring, req, pos, last_pos[t], taps - 1, channels, blockIdx.y, gridDim.y, threadIdx.x, blockDim.x);
  const float* x = o + t * inner + c0;
  const A* z = p + z_off + c0;
  float ss = 0.f;
  const bool vec = sizeof(A) == 2 && ((part | ldp | ldo | z_off) & 3) == 0 && (inner & 3) == 0;
  if (vec) {
    for (int c = threadIdx.x * 4; c < part; c += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(x + c);
      const uint2 u = *reinterpret_cast<const uint2*>(z + c);
      const float2 z0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
      const float2 z1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
      const float4 y = make_float4(v.x * silu_bf16(z0.x), v.y * silu_bf16(z0.y),
                                   v.z * silu_bf16(z1.x), v.w * silu_bf16(z1.y));
      *reinterpret_cast<float4*>(row + c) = y;
      ss = fmaf(y.x, y.x, fmaf(y.y, y.y, fmaf(y.z, y.z, fmaf(y.w, y.w, ss))));
    }
  } else {
    for (int c = threadIdx.x; c < part; c += blockDim.x) {
      const float y = x[c] * silu_f(ld_act(z + c));
      row[c] = y;
      ss = fmaf(y, y, ss);
    }
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / static_cast<float>(part) + eps);
  if (vec) {
    for (int c = threadIdx.x * 4; c < part; c += blockDim.x * 4) {
      const float4 y = *reinterpret_cast<const float4*>(row + c), g = *reinterpret_cast<const float4*>(w + c0 + c);
      uint2 pk;
      *reinterpret_cast<__nv_bfloat162*>(&pk.x) = __floats2bfloat162_rn(y.x * r * g.x, y.y * r * g.y);
      *reinterpret_cast<__nv_bfloat162*>(&pk.y) = __floats2bfloat162_rn(y.z * r * g.z, y.w * r * g.w);
      *reinterpret_cast<uint2*>(to + c0 + c) = pk;
    }
  } else {
    for (int c = threadIdx.x; c < part; c += blockDim.x) st_act(to + c0 + c, row[c] * r * w[c0 + c]);
  }
}

}  // namespace stk

using namespace stk;

// Spans of min_span .. max_span tokens, token by token, over the operands of stk_mamba2_conv.
STK_API int stk_mamba2_scan(const void* xbc, long long ld, const float* steps, const float* skip, const int* query_start,
                            const int* req_rows, const int* start_pos, int n_req, float* S, float* o, int heads, int state, int vdim,
                            int groups, int fp32, int min_span, int max_span, int T, void* stream) {
  if (T <= 0) return 0;
  if (groups < 1 || heads % groups) return -1;
  const ScanArgs a{query_start, req_rows, start_pos, n_req, S, o, heads, state, vdim};
  const int inner = heads * vdim, hpg = heads / groups;
  if (fp32)
    return launch_scan(Mamba2Front<float>{(const float*)xbc, ld, steps, state, vdim, inner, groups, hpg, heads, T, skip}, a, min_span,
                       max_span, (cudaStream_t)stream);
  return launch_scan(Mamba2Front<__nv_bfloat16>{(const __nv_bfloat16*)xbc, ld, steps, state, vdim, inner, groups, hpg, heads, T, skip}, a,
                     min_span, max_span, (cudaStream_t)stream);
}

// out [T, ldo] in the compute type: convolved channels, zeros up to ldo (a multiple of 8); steps fp32 [2, heads, T]: log decays, step
// sizes.
STK_API int stk_mamba2_conv(const void* proj, long long ldp, int x_off, int dt_off, const float* taps, const float* conv_bias, int n_taps,
                            const void* ring, const float* dt_bias, const float* neg_a, const int64_t* positions, const int* tok_req,
                            const int* first_pos, void* out, long long ldo, float* steps, int heads, int channels, int fp32, int T,
                            void* stream) {
  if (T <= 0) return 0;
  if (n_taps < 1 || ldo % 8 || ldo < channels || (reinterpret_cast<uintptr_t>(out) & 15)) return -1;
  const ConvArgs c{proj, ldp, x_off, dt_off, taps, conv_bias, n_taps, ring, dt_bias, neg_a, channels};
  const int vec = channels % kConvCh == 0 && ldp % kConvCh == 0 && x_off % kConvCh == 0 &&
                  ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(ring) | reinterpret_cast<uintptr_t>(taps) |
                    reinterpret_cast<uintptr_t>(conv_bias)) & 15) == 0;
  const bool few = T <= 256;                               // one token per thread
  const int tok = few ? 1 : kConvTok;
  constexpr int kBlock = kConvThreads * kConvCh;
  const dim3 grid(static_cast<unsigned>((ldo + kBlock - 1) / kBlock + 1), (T + tok - 1) / tok);
  cudaStream_t st = (cudaStream_t)stream;
#define STK_CONV(A, N)                                                                                                               \
  if (few) launch_pdl(mamba2_conv_kernel<A, N, 1>, grid, dim3(kConvThreads), 0, st, c, positions, tok_req, first_pos, (A*)out, ldo, steps, heads, T, vec); \
  else launch_pdl(mamba2_conv_kernel<A, N, kConvTok>, grid, dim3(kConvThreads), 0, st, c, positions, tok_req, first_pos, (A*)out, ldo, steps, heads, T, vec)
  if (fp32) {
    STK_CONV(float, 0);
  } else {
    switch (n_taps) {
      case 2: STK_CONV(__nv_bfloat16, 2); break;
      case 3: STK_CONV(__nv_bfloat16, 3); break;
      case 4: STK_CONV(__nv_bfloat16, 4); break;
      default: STK_CONV(__nv_bfloat16, 0); break;
    }
  }
#undef STK_CONV
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_mamba2_finish(const float* o, const void* proj, long long ldp, int z_off, int x_off, int channels, const float* norm_w,
                              float eps, int norm_groups, const int* tok_req, const int64_t* positions, const int* last_pos, void* ring,
                              int n_taps, void* out, long long ldo, int cols, int fp32, int inner, int T, void* stream) {
  if (T <= 0) return 0;
  if (norm_groups < 1 || inner % norm_groups || n_taps < 1 || norm_groups > 65535) return -1;
  const int part = inner / norm_groups;
  const size_t smem = static_cast<size_t>(part) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  if (smem > 40 * 1024 &&
      (cudaFuncSetAttribute(mamba2_finish_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess ||
       cudaFuncSetAttribute(mamba2_finish_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess))
    return -3;
  const dim3 grid(T, norm_groups);
  cudaStream_t st = (cudaStream_t)stream;
  if (!fp32 && part <= 1024 && part % 4 == 0 && ldp % 4 == 0 && ldo % 4 == 0 && z_off % 4 == 0 &&
      ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(out)) & 7) == 0) {
    const dim3 warps(static_cast<unsigned>((static_cast<long long>(T) * norm_groups + 7) / 8));
#define STK_FINISH(NV)                                                                                                             \
  launch_pdl(mamba2_finish_warp_kernel<NV>, warps, dim3(256), 0, st, o, (const __nv_bfloat16*)proj, ldp, z_off, x_off, channels, norm_w, \
             eps, tok_req, positions, last_pos, (__nv_bfloat16*)ring, n_taps, (__nv_bfloat16*)out, ldo, cols, inner, part, norm_groups, T)
    if (part <= 256) STK_FINISH(2);
    else if (part <= 512) STK_FINISH(4);
    else STK_FINISH(8);
#undef STK_FINISH
    return cudaGetLastError() == cudaSuccess ? 0 : -4;
  }
  if (fp32)
    launch_pdl(mamba2_finish_kernel<float>, grid, dim3(256), smem, st, o, (const float*)proj, ldp, z_off, x_off, channels, norm_w, eps,
               tok_req, positions, last_pos, (float*)ring, n_taps, (float*)out, ldo, cols, inner, part);
  else
    launch_pdl(mamba2_finish_kernel<__nv_bfloat16>, grid, dim3(256), smem, st, o, (const __nv_bfloat16*)proj, ldp, z_off, x_off, channels,
               norm_w, eps, tok_req, positions, last_pos, (__nv_bfloat16*)ring, n_taps, (__nv_bfloat16*)out, ldo, cols, inner, part);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
