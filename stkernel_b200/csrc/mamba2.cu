// Mamba-2: a linear recurrence (linear_scan.cuh) with k = dt B, q = C, v = x and log decay -exp(A) dt, whose operands x, B and C come
// through a short causal convolution per channel and silu.
//
//   mamba2_scan        decode rows, short spans, float32: convolution and step size on the way into the recurrence
//   mamba2_conv        long spans: convolved operands in bf16, step sizes and log decays for the chunked form
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

// Channel ch of token t, the i-th of its span, at position pos.
template <typename A>
__device__ __forceinline__ float conv_at(const ConvArgs& a, long long t, int i, long long pos, long long row, int ch) {
  const A* x = reinterpret_cast<const A*>(a.proj) + t * a.ldp + a.x_off + ch;
  const int keep = a.n - 1;
  float s = a.bias[ch];
  for (int j = 0; j < a.n; ++j) {
    float in = 0.f;
    if (j <= i) in = ld_act(x - j * a.ldp);
    else if (pos >= j) in = ld_act(reinterpret_cast<const A*>(a.ring) + (row * keep + (pos - j) % keep) * a.channels + ch);
    s = fmaf(a.taps[(a.n - 1 - j) * a.channels + ch], in, s);
  }
  return silu_f(s);
}

template <typename A>
struct Mamba2Front {
  static constexpr bool kValues = true;
  ConvArgs c;
  int N, V, inner, groups, hpg;
  const float* skips;
  __device__ __forceinline__ float skip(int h) const { return skips[h]; }
  __device__ __forceinline__ float value(long long, int, int) const { return 0.f; }
  __device__ __forceinline__ float2 fill(long long t, int i, long long pos, long long row, int h, int col0, int cols, float* q, float* k,
                                         float* x) const {
    const float dt = softplus_f(ld_act(reinterpret_cast<const A*>(c.proj) + t * c.ldp + c.dt_off + h) + c.dt_bias[h]);
    const int g = h / hpg, b0 = inner + g * N, c0 = inner + (groups + g) * N;
    for (int e = threadIdx.x; e < 2 * N + cols; e += kScanThreads) {
      if (e < N) q[e] = conv_at<A>(c, t, i, pos, row, c0 + e);
      else if (e < 2 * N) k[e - N] = conv_at<A>(c, t, i, pos, row, b0 + e - N) * dt;
      else x[e - 2 * N] = conv_at<A>(c, t, i, pos, row, h * V + col0 + e - 2 * N);
    }
    // slow decays as 1 and the (small) difference from it: a rounded factor close to 1 would be off in the same direction for long
    const float lg = c.neg_a[h] * dt;
    return lg > -0.25f ? make_float2(1.f, expm1f(lg)) : make_float2(expf(lg), 0.f);
  }
};

constexpr int kConvTok = 8;

// Eight channels x kConvTok tokens per thread; the inputs slide through registers where the taps are few (NT), otherwise they are
// read again for every tap.  The grid's last column of blocks forms the step sizes.
template <int NT>
__global__ void __launch_bounds__(128)
mamba2_conv_kernel(const ConvArgs a, const int64_t* __restrict__ positions, const int* __restrict__ tok_req,
                   const int* __restrict__ first_pos, __nv_bfloat16* __restrict__ out, long long ldo, float* __restrict__ steps, int H,
                   int T, int vec) {
  pdl_wait();
  pdl_trigger();
  const __nv_bfloat16* proj = reinterpret_cast<const __nv_bfloat16*>(a.proj);
  if (blockIdx.x == gridDim.x - 1) {
    // steps [0][H][T]: log decays, [1][H][T]: input weights
    for (int e = threadIdx.x; e < kConvTok * H; e += 128) {
      const int h = e / kConvTok, t = blockIdx.y * kConvTok + e % kConvTok;
      if (t >= T) continue;
      const float dt = softplus_f(bf16_to_f(proj[t * a.ldp + a.dt_off + h]) + a.dt_bias[h]);
      steps[static_cast<long long>(h) * T + t] = dt * a.neg_a[h];
      steps[(static_cast<long long>(H) + h) * T + t] = dt;
    }
    return;
  }
  const int ch = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (ch >= ldo) return;
  const int nc = min(8, a.channels - ch), t0 = blockIdx.y * kConvTok, keep = a.n - 1;
  const __nv_bfloat16* ring = reinterpret_cast<const __nv_bfloat16*>(a.ring);
  // input j tokens before token t: its own span's row, the ring, or zero
  auto input = [&](int t, int j, float (&f)[8]) {
    const int first = first_pos[t];
    const long long pos = positions[t];
    const __nv_bfloat16* src = nullptr;
    if (pos - j >= first) src = proj + (t - j) * a.ldp + a.x_off + ch;
    else if (pos >= j) src = ring + (static_cast<long long>(tok_req[t]) * keep + (pos - j) % keep) * a.channels + ch;
    if (src != nullptr && vec) {
      const uint4 v = *reinterpret_cast<const uint4*>(src);
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const float2 u = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&v)[c]);
        f[2 * c] = u.x;
        f[2 * c + 1] = u.y;
      }
    } else {
#pragma unroll
      for (int c = 0; c < 8; ++c) f[c] = src != nullptr && c < nc ? bf16_to_f(src[c]) : 0.f;
    }
  };
  float w[NT > 0 ? NT : 1][8], bias[8];
#pragma unroll
  for (int c = 0; c < 8; ++c) bias[c] = c < nc ? a.bias[ch + c] : 0.f;
  if (NT > 0) {
#pragma unroll
    for (int j = 0; j < (NT > 0 ? NT : 1); ++j)
#pragma unroll
      for (int c = 0; c < 8; ++c) w[j][c] = c < nc ? a.taps[(a.n - 1 - j) * a.channels + ch + c] : 0.f;
  }
  float past[NT > 0 ? NT : 1][8];                       // past[j]: input j tokens before the current one
  int prev_req = -2;
  long long prev_pos = -2;
  for (int t = t0; t < min(T, t0 + kConvTok); ++t) {
    const int req = tok_req[t];
    const long long pos = positions[t];
    float s[8];
#pragma unroll
    for (int c = 0; c < 8; ++c) s[c] = bias[c];
    if (req >= 0 && pos >= 0) {
      if (NT > 0) {
        constexpr int kN = NT > 0 ? NT : 1;
        if (req == prev_req && pos == prev_pos + 1) {
#pragma unroll
          for (int j = kN - 1; j > 0; --j)
#pragma unroll
            for (int c = 0; c < 8; ++c) past[j][c] = past[j - 1][c];
        } else {
#pragma unroll
          for (int j = 1; j < kN; ++j) input(t, j, past[j]);
        }
        input(t, 0, past[0]);
#pragma unroll
        for (int j = 0; j < kN; ++j)
#pragma unroll
          for (int c = 0; c < 8; ++c) s[c] = fmaf(w[j][c], past[j][c], s[c]);
      } else {
        for (int j = 0; j < a.n; ++j) {
          float f[8];
          input(t, j, f);
#pragma unroll
          for (int c = 0; c < 8; ++c)
            if (c < nc) s[c] = fmaf(a.taps[(a.n - 1 - j) * a.channels + ch + c], f[c], s[c]);
        }
      }
    }
    prev_req = req;
    prev_pos = pos;
    __align__(16) __nv_bfloat162 b[4];
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const float x = s[2 * c], y = s[2 * c + 1];
      b[c] = __floats2bfloat162_rn(2 * c < nc ? x / (1.f + __expf(-x)) : 0.f, 2 * c + 1 < nc ? y / (1.f + __expf(-y)) : 0.f);
    }
    *reinterpret_cast<uint4*>(out + t * ldo + ch) = *reinterpret_cast<const uint4*>(b);
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
  const int keep = taps - 1;
  if (keep > 0 && pos > last_pos[t] - keep) {
    A* dst = ring + (static_cast<long long>(req) * keep + pos % keep) * channels;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < channels; c += gridDim.y * blockDim.x) dst[c] = p[x_off + c];
  }
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
      const float4 y = make_float4(v.x * z0.x / (1.f + __expf(-z0.x)), v.y * z0.y / (1.f + __expf(-z0.y)),
                                   v.z * z1.x / (1.f + __expf(-z1.x)), v.w * z1.y / (1.f + __expf(-z1.y)));
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

// Spans of min_span .. max_span tokens, token by token.
STK_API int stk_mamba2_scan(const void* proj, long long ldp, int x_off, int dt_off, const float* taps, const float* conv_bias, int n_taps,
                            const void* ring, const float* dt_bias, const float* neg_a, const float* skip, const int* query_start,
                            const int* req_rows, const int* start_pos, int n_req, float* S, float* o, int heads, int state, int vdim,
                            int groups, int fp32, int min_span, int max_span, int T, void* stream) {
  if (T <= 0) return 0;
  if (n_taps < 1 || groups < 1 || heads % groups) return -1;
  const ScanArgs a{query_start, req_rows, start_pos, n_req, S, o, heads, state, vdim};
  const int inner = heads * vdim;
  const ConvArgs c{proj, ldp, x_off, dt_off, taps, conv_bias, n_taps, ring, dt_bias, neg_a, inner + 2 * groups * state};
  if (fp32)
    return launch_scan(Mamba2Front<float>{c, state, vdim, inner, groups, heads / groups, skip}, a, min_span, max_span, (cudaStream_t)stream);
  return launch_scan(Mamba2Front<__nv_bfloat16>{c, state, vdim, inner, groups, heads / groups, skip}, a, min_span, max_span,
                     (cudaStream_t)stream);
}

// bf16.  out [T, ldo]: convolved channels, zeros up to ldo (a multiple of 8); steps fp32 [2, heads, T]: log decays, step sizes.
STK_API int stk_mamba2_conv(const void* proj, long long ldp, int x_off, int dt_off, const float* taps, const float* conv_bias, int n_taps,
                            const void* ring, const float* dt_bias, const float* neg_a, const int64_t* positions, const int* tok_req,
                            const int* first_pos, void* out, long long ldo, float* steps, int heads, int channels, int T, void* stream) {
  if (T <= 0) return 0;
  if (n_taps < 1 || ldo % 8 || ldo < channels || (reinterpret_cast<uintptr_t>(out) & 15)) return -1;
  const ConvArgs c{proj, ldp, x_off, dt_off, taps, conv_bias, n_taps, ring, dt_bias, neg_a, channels};
  const int vec = channels % 8 == 0 && ldp % 8 == 0 && x_off % 8 == 0 &&
                  ((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(ring)) & 15) == 0;
  const dim3 grid(static_cast<unsigned>((ldo + 1023) / 1024 + 1), (T + kConvTok - 1) / kConvTok);
  cudaStream_t st = (cudaStream_t)stream;
#define STK_CONV(N) \
  launch_pdl(mamba2_conv_kernel<N>, grid, dim3(128), 0, st, c, positions, tok_req, first_pos, (__nv_bfloat16*)out, ldo, steps, heads, T, vec)
  switch (n_taps) {
    case 2: STK_CONV(2); break;
    case 3: STK_CONV(3); break;
    case 4: STK_CONV(4); break;
    default: STK_CONV(0); break;
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
  if (fp32)
    launch_pdl(mamba2_finish_kernel<float>, grid, dim3(256), smem, st, o, (const float*)proj, ldp, z_off, x_off, channels, norm_w, eps,
               tok_req, positions, last_pos, (float*)ring, n_taps, (float*)out, ldo, cols, inner, part);
  else
    launch_pdl(mamba2_finish_kernel<__nv_bfloat16>, grid, dim3(256), smem, st, o, (const __nv_bfloat16*)proj, ldp, z_off, x_off, channels,
               norm_w, eps, tok_req, positions, last_pos, (__nv_bfloat16*)ring, n_taps, (__nv_bfloat16*)out, ldo, cols, inner, part);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
