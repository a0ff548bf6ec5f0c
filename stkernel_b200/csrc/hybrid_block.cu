// Residual-side kernels of the layer-by-layer decoders (models/hybrid.py): scaled embedding into an fp32 residual, residual add
// fused with the next norm (parallel block), norm of a sublayer's output fused with the residual add (post-norm block), the update
// of several residual streams fused with the norm of their next weighted sum (streams block), and the feed-forward half of the
// joined sublayer buffer.
#define STK_PDL_CLASS 4
#include "hybrid_block.cuh"
#include "pairs.cuh"

namespace stk {

// h != nullptr: the row also in the compute type E, zero-padded to `width` columns.  copies: the row that many times, W apart.
template <typename E>
__global__ void __launch_bounds__(256)
embed_scaled_kernel(const int64_t* __restrict__ ids, const E* __restrict__ embed, float* __restrict__ x, long long ldx, int copies, int W,
                    int vocab, float scale, E* __restrict__ h, long long ldh, int width, int* status) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  const long long id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0) set_status(status, kBadIndex, t);
  const bool vec = sizeof(E) == 2 && (W & 7) == 0 && (ldx & 3) == 0 && (ldh & 7) == 0;
  if (h != nullptr)
    for (int i = (vec ? W : 0) + threadIdx.x; i < width; i += blockDim.x)
      st_act(h + t * ldh + i, ok && i < W ? ld_act(embed + id * W + i) * scale : 0.f);
  if (vec) {
    for (int i = threadIdx.x * 8; i < W; i += blockDim.x * 8) {
      uint4 v = make_uint4(0, 0, 0, 0);
      if (ok) v = __ldg(reinterpret_cast<const uint4*>(embed + id * W + i));
      float2 f[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) f[j] = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&v)[j]);
      for (int c = 0; c < copies; ++c) {
        float* to = x + t * ldx + c * W + i;
        *reinterpret_cast<float4*>(to) = make_float4(f[0].x * scale, f[0].y * scale, f[1].x * scale, f[1].y * scale);
        *reinterpret_cast<float4*>(to + 4) = make_float4(f[2].x * scale, f[2].y * scale, f[3].x * scale, f[3].y * scale);
      }
      if (h != nullptr) {
        __align__(16) __nv_bfloat162 b[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) b[j] = __floats2bfloat162_rn(f[j].x * scale, f[j].y * scale);
        *reinterpret_cast<uint4*>(reinterpret_cast<__nv_bfloat16*>(h) + t * ldh + i) = *reinterpret_cast<const uint4*>(b);
      }
    }
    return;
  }
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    const float v = ok ? ld_act(embed + id * W + i) * scale : 0.f;
    for (int c = 0; c < copies; ++c) x[t * ldx + c * W + i] = v;
  }
}

// x[r] += y[r]; h[t] = norm(x[r]) * w with r = rows ? rows[t] : t (with `rows` the sum is not written back).  The
// row stays in shared memory between the three passes (mean, squared deviations, output), all in fp32.  center: layer norm,
// otherwise RMS norm (no mean).
template <typename O>
__global__ void __launch_bounds__(1024)
add_layer_norm_kernel(float* __restrict__ x, long long ldx, const float* __restrict__ y, long long ldy,
                      const float* __restrict__ w, O* __restrict__ h, long long ldh, int W, int width, float eps,
                      const int64_t* __restrict__ rows, int center) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const long long r = rows != nullptr ? rows[blockIdx.x] : static_cast<long long>(blockIdx.x);
  float* xr = x + r * ldx;
  const float* yr = y != nullptr ? y + r * ldy : nullptr;
  const bool store = yr != nullptr && rows == nullptr;
  float s = 0.f;
  if ((W & 3) == 0 && (ldx & 3) == 0 && (ldy & 3) == 0) {
    for (int i = threadIdx.x * 4; i < W; i += blockDim.x * 4) {
      float4 v = *reinterpret_cast<const float4*>(xr + i);
      if (yr != nullptr) {
        const float4 u = *reinterpret_cast<const float4*>(yr + i);
        v.x += u.x; v.y += u.y; v.z += u.z; v.w += u.w;
        if (store) *reinterpret_cast<float4*>(xr + i) = v;
      }
      *reinterpret_cast<float4*>(row + i) = v;
      s += (v.x + v.y) + (v.z + v.w);
    }
  } else {
    for (int i = threadIdx.x; i < W; i += blockDim.x) {
      float v = xr[i];
      if (yr != nullptr) {
        v += yr[i];
        if (store) xr[i] = v;
      }
      row[i] = v;
      s += v;
    }
  }
  s = block_sum(s, red);                                  // also publishes the row
  const float mean = center ? s / static_cast<float>(W) : 0.f;
  float q = 0.f;
  for (int i = threadIdx.x; i < W; i += blockDim.x) {
    const float d = row[i] - mean;
    q = fmaf(d, d, q);
  }
  const float inv = 1.f / sqrtf(block_sum(q, red) / static_cast<float>(W) + eps);
  O* hr = h + blockIdx.x * ldh;
  if (sizeof(O) == 2 && (width & 1) == 0 && (ldh & 1) == 0) {
    for (int i = threadIdx.x * 2; i < width; i += blockDim.x * 2) {
      const float a = i < W ? (row[i] - mean) * inv * w[i] : 0.f;
      const float b = i + 1 < W ? (row[i + 1] - mean) * inv * w[i + 1] : 0.f;
      *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<__nv_bfloat16*>(hr) + i) = __floats2bfloat162_rn(a, b);
    }
  } else {
    for (int i = threadIdx.x; i < width; i += blockDim.x) st_act(hr + i, i < W ? (row[i] - mean) * inv * w[i] : 0.f);
  }
}

// x[t] += rms_norm(y[t]) * w and h[t] = x[t] in the compute type, zero-padded to `width` columns (h may be null).  y is either
// one fp32 row per token, or the weighted sum of `top` expert rows: row pair_row[t * top + j] (t * top + j when pair_row is
// null) times weights[t * top + j].
template <typename A>
struct PostNormArgs {
  float* x; long long ldx;
  const float* y; long long ldy;
  const A* pairs; long long ldp; const int* pair_row; const float* weights; int top;
  const float* w; float eps;
  A* h; long long ldh;
  int W, width;
};

template <typename A>
__global__ void __launch_bounds__(1024)
post_norm_add_kernel(const PostNormArgs<A> a) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  __shared__ long long src[32];
  __shared__ float wt[32];
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  float q = 0.f;
  if (a.pairs != nullptr) {
    if (static_cast<int>(threadIdx.x) < a.top) {
      const long long p = t * a.top + threadIdx.x;
      const int r = a.pair_row != nullptr ? a.pair_row[p] : static_cast<int>(p);
      src[threadIdx.x] = r < 0 ? 0 : r * a.ldp;
      wt[threadIdx.x] = r < 0 ? 0.f : a.weights[p];
    }
    __syncthreads();
    if (sizeof(A) == 2 && (a.W & 7) == 0 && (a.ldp & 7) == 0) {
      for (int i = threadIdx.x * 8; i < a.W; i += blockDim.x * 8) {
        float s[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) s[k] = 0.f;
        for (int j = 0; j < a.top; ++j) {
          const uint4 v = *reinterpret_cast<const uint4*>(a.pairs + src[j] + i);
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float2 f = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&v)[k]);
            s[2 * k] = fmaf(wt[j], f.x, s[2 * k]);
            s[2 * k + 1] = fmaf(wt[j], f.y, s[2 * k + 1]);
          }
        }
#pragma unroll
        for (int k = 0; k < 8; ++k) q = fmaf(s[k], s[k], q);
        *reinterpret_cast<float4*>(row + i) = make_float4(s[0], s[1], s[2], s[3]);
        *reinterpret_cast<float4*>(row + i + 4) = make_float4(s[4], s[5], s[6], s[7]);
      }
    } else {
      for (int i = threadIdx.x; i < a.W; i += blockDim.x) {
        float s = 0.f;
        for (int j = 0; j < a.top; ++j) s = fmaf(wt[j], ld_act(a.pairs + src[j] + i), s);
        row[i] = s;
        q = fmaf(s, s, q);
      }
    }
  } else if ((a.W & 3) == 0 && (a.ldy & 3) == 0) {
    for (int i = threadIdx.x * 4; i < a.W; i += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(a.y + t * a.ldy + i);
      *reinterpret_cast<float4*>(row + i) = v;
      q = fmaf(v.x, v.x, q); q = fmaf(v.y, v.y, q); q = fmaf(v.z, v.z, q); q = fmaf(v.w, v.w, q);
    }
  } else {
    for (int i = threadIdx.x; i < a.W; i += blockDim.x) {
      const float v = a.y[t * a.ldy + i];
      row[i] = v;
      q = fmaf(v, v, q);
    }
  }
  const float inv = 1.f / sqrtf(block_sum(q, red) / static_cast<float>(a.W) + a.eps);
  float* xr = a.x + t * a.ldx;
  A* hr = a.h != nullptr ? a.h + t * a.ldh : nullptr;
  if ((a.W & 3) == 0 && (a.ldx & 3) == 0 && (a.ldh & 3) == 0) {
    for (int i = threadIdx.x * 4; i < a.W; i += blockDim.x * 4) {
      float4 v = *reinterpret_cast<const float4*>(xr + i);
      const float4 r = *reinterpret_cast<const float4*>(row + i);
      const float4 w = *reinterpret_cast<const float4*>(a.w + i);
      v.x = fmaf(r.x * inv, w.x, v.x);
      v.y = fmaf(r.y * inv, w.y, v.y);
      v.z = fmaf(r.z * inv, w.z, v.z);
      v.w = fmaf(r.w * inv, w.w, v.w);
      *reinterpret_cast<float4*>(xr + i) = v;
      if (hr != nullptr) {
        if (sizeof(A) == 2) {
          __align__(8) __nv_bfloat162 b[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
          *reinterpret_cast<uint2*>(hr + i) = *reinterpret_cast<const uint2*>(b);
        } else {
          *reinterpret_cast<float4*>(hr + i) = v;
        }
      }
    }
    if (hr != nullptr)
      for (int i = a.W + threadIdx.x; i < a.width; i += blockDim.x) st_act(hr + i, 0.f);
    return;
  }
  for (int i = threadIdx.x; i < (hr != nullptr ? a.width : a.W); i += blockDim.x) {
    float v = 0.f;
    if (i < a.W) {
      v = fmaf(row[i] * inv, a.w[i], xr[i]);
      xr[i] = v;
    }
    if (hr != nullptr) st_act(hr + i, v);
  }
}

// Streams x [*, S, W] fp32: x_t <- sum_s mix[s, t] x_s + write[t] y (y as in PostNormArgs, none at all if both are null), then
// h = layer norm (weight w, bias b) of u = sum_s read[s] x_s, in the compute type, zero-padded to `width` columns.  rows: only these
// rows, and the streams stay as they were.
template <typename A>
struct StreamArgs {
  float* x;
  const float* y; long long ldy;
  const A* pairs; long long ldp; const int* pair_row; const float* weights; int top;
  const float* mix; const float* write; const float* read;
  const float* w; const float* b; float eps;
  A* h; long long ldh;
  int W, width;
  const int64_t* rows;
};

// N consecutive columns of one row in all streams, before their update.
template <int S, int N>
__device__ __forceinline__ void load_streams(const float* xr, int W, int i, float (&v)[S][N]) {
#pragma unroll
  for (int s = 0; s < S; ++s) {
    if constexpr (N == 4) {
      const float4 f = *reinterpret_cast<const float4*>(xr + s * W + i);
      v[s][0] = f.x; v[s][1] = f.y; v[s][2] = f.z; v[s][3] = f.w;
    } else {
      v[s][0] = xr[s * W + i];
    }
  }
}

// The same columns of the sublayer's output.
template <typename A, int N>
__device__ __forceinline__ void load_output(const StreamArgs<A>& a, long long r, int i, const long long* src, const float* wt, float (&y)[N]) {
#pragma unroll
  for (int k = 0; k < N; ++k) y[k] = 0.f;
  if (a.pairs != nullptr) {
    if constexpr (N == 4 && sizeof(A) == 2) {
      for (int j0 = 0; j0 < a.top; j0 += 4) {                     // four rows in flight
        uint2 q[4];
#pragma unroll
        for (int j = 0; j < 4; ++j)
          q[j] = j0 + j < a.top ? *reinterpret_cast<const uint2*>(a.pairs + src[j0 + j] + i) : make_uint2(0, 0);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float w = j0 + j < a.top ? wt[j0 + j] : 0.f;
          const float2 f0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q[j].x));
          const float2 f1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q[j].y));
          y[0] = fmaf(w, f0.x, y[0]); y[1] = fmaf(w, f0.y, y[1]);
          y[2] = fmaf(w, f1.x, y[2]); y[3] = fmaf(w, f1.y, y[3]);
        }
      }
    } else {
      for (int j = 0; j < a.top; ++j)
#pragma unroll
        for (int k = 0; k < N; ++k) y[k] = fmaf(wt[j], ld_act(a.pairs + src[j] + i + k), y[k]);
    }
  } else if constexpr (N == 4) {
    const float4 f = *reinterpret_cast<const float4*>(a.y + r * a.ldy + i);
    y[0] = f.x; y[1] = f.y; y[2] = f.z; y[3] = f.w;
  } else {
    y[0] = a.y[r * a.ldy + i];
  }
}

// Streams after the update (stored if `store`) and u = sum_s read[s] x_s.
template <int S, int N>
__device__ __forceinline__ void mix_streams(float* xr, int W, int i, const float (&v)[S][N], const float (&y)[N], const float (&mix)[S][S],
                                            const float (&write)[S], const float (&read)[S], float (&u)[N], bool has_y, bool store) {
#pragma unroll
  for (int k = 0; k < N; ++k) u[k] = 0.f;
#pragma unroll
  for (int t = 0; t < S; ++t) {
    float n[N];
#pragma unroll
    for (int k = 0; k < N; ++k) {
      if (has_y) {
        n[k] = write[t] * y[k];
#pragma unroll
        for (int s = 0; s < S; ++s) n[k] = fmaf(mix[s][t], v[s][k], n[k]);
      } else {
        n[k] = v[t][k];
      }
      u[k] = fmaf(read[t], n[k], u[k]);
    }
    if (store) {
      if constexpr (N == 4) *reinterpret_cast<float4*>(xr + t * W + i) = make_float4(n[0], n[1], n[2], n[3]);
      else xr[t * W + i] = n[0];
    }
  }
}

// NIT > 0: a thread's NIT groups of four columns stay in registers (W a multiple of 4, at most NIT * 4 * blockDim.x); 0: any width, the
// row in shared memory.
template <typename A, int S, int NIT>
__global__ void __launch_bounds__(1024)
stream_norm_kernel(const StreamArgs<A> a) {
  extern __shared__ __align__(16) float row[];
  __shared__ float red[32];
  __shared__ long long src[32];
  __shared__ float wt[32];
  pdl_wait();
  pdl_trigger();
  const long long r = a.rows != nullptr ? a.rows[blockIdx.x] : static_cast<long long>(blockIdx.x);
  const bool has_y = a.y != nullptr || a.pairs != nullptr, store = has_y && a.rows == nullptr;
  if (a.pairs != nullptr && static_cast<int>(threadIdx.x) < a.top) {
    const long long p = r * a.top + threadIdx.x;
    const int at = a.pair_row != nullptr ? a.pair_row[p] : static_cast<int>(p);
    src[threadIdx.x] = at < 0 ? 0 : at * a.ldp;
    wt[threadIdx.x] = at < 0 ? 0.f : a.weights[p];
  }
  float mix[S][S], write[S], read[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    read[s] = a.read[s];
    write[s] = has_y ? a.write[s] : 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = has_y ? a.mix[s * S + t] : 0.f;
  }
  float* xr = a.x + r * S * a.W;
  A* hr = a.h + blockIdx.x * a.ldh;
  const float n = static_cast<float>(a.W);
  if constexpr (NIT > 0) {
    float u[NIT][4], sum = 0.f;
    float4 w = make_float4(0.f, 0.f, 0.f, 0.f), b = w;
    float v[S][4], y[4];
    const int i0 = threadIdx.x * 4;
    if (i0 < a.W) {                                                      // before the wait for the expert rows' places
      load_streams<S, 4>(xr, a.W, i0, v);
      if (NIT == 1) {
        w = *reinterpret_cast<const float4*>(a.w + i0);
        b = *reinterpret_cast<const float4*>(a.b + i0);
      }
    }
    if (a.pairs != nullptr) __syncthreads();
#pragma unroll
    for (int e = 0; e < NIT; ++e) {
      const int i = i0 + e * blockDim.x * 4;
      if (i < a.W) {
        if (e > 0) load_streams<S, 4>(xr, a.W, i, v);
        if (has_y) load_output<A, 4>(a, r, i, src, wt, y);
        mix_streams<S, 4>(xr, a.W, i, v, y, mix, write, read, u[e], has_y, store);
        sum += (u[e][0] + u[e][1]) + (u[e][2] + u[e][3]);
      } else {
#pragma unroll
        for (int k = 0; k < 4; ++k) u[e][k] = 0.f;
      }
    }
    const float mean = block_sum(sum, red) / n;
    float q = 0.f;
#pragma unroll
    for (int e = 0; e < NIT; ++e)
      if (i0 + e * static_cast<int>(blockDim.x) * 4 < a.W) {
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          u[e][k] -= mean;
          q = fmaf(u[e][k], u[e][k], q);
        }
      }
    const float inv = 1.f / sqrtf(block_sum(q, red) / n + a.eps);
#pragma unroll
    for (int e = 0; e < NIT; ++e) {
      const int i = i0 + e * blockDim.x * 4;
      if (i >= a.W) continue;
      if (NIT > 1) {
        w = *reinterpret_cast<const float4*>(a.w + i);
        b = *reinterpret_cast<const float4*>(a.b + i);
      }
      const float o[4] = {fmaf(u[e][0] * inv, w.x, b.x), fmaf(u[e][1] * inv, w.y, b.y), fmaf(u[e][2] * inv, w.z, b.z),
                          fmaf(u[e][3] * inv, w.w, b.w)};
      if (sizeof(A) == 2 && (a.ldh & 3) == 0) {
        __align__(8) __nv_bfloat162 pk[2] = {__floats2bfloat162_rn(o[0], o[1]), __floats2bfloat162_rn(o[2], o[3])};
        *reinterpret_cast<uint2*>(hr + i) = *reinterpret_cast<const uint2*>(pk);
      } else {
#pragma unroll
        for (int k = 0; k < 4; ++k) st_act(hr + i + k, o[k]);
      }
    }
    for (int i = a.W + threadIdx.x; i < a.width; i += blockDim.x) st_act(hr + i, 0.f);
  } else {
    if (a.pairs != nullptr) __syncthreads();
    float sum = 0.f;
    for (int i = threadIdx.x; i < a.W; i += blockDim.x) {
      float v[S][1], y[1], u[1];
      load_streams<S, 1>(xr, a.W, i, v);
      if (has_y) load_output<A, 1>(a, r, i, src, wt, y);
      mix_streams<S, 1>(xr, a.W, i, v, y, mix, write, read, u, has_y, store);
      row[i] = u[0];
      sum += u[0];
    }
    const float mean = block_sum(sum, red) / n;                          // also publishes the row
    float q = 0.f;
    for (int i = threadIdx.x; i < a.W; i += blockDim.x) {
      const float d = row[i] - mean;
      q = fmaf(d, d, q);
    }
    const float inv = 1.f / sqrtf(block_sum(q, red) / n + a.eps);
    for (int i = threadIdx.x; i < a.width; i += blockDim.x)
      st_act(hr + i, i < a.W ? fmaf((row[i] - mean) * inv, a.w[i], a.b[i]) : 0.f);
  }
}

template <typename A, int S>
static int launch_stream_norm(const StreamArgs<A>& a, int T, cudaStream_t st) {
  const int threads = T > 148 || a.W <= 1024 ? 256 : (a.W <= 2048 ? 512 : 1024);
  const int its = a.W % 4 == 0 && a.ldy % 4 == 0 && a.ldp % 4 == 0 ? (a.W / 4 + threads - 1) / threads : 99;
  if (its == 1) launch_pdl(stream_norm_kernel<A, S, 1>, dim3(T), dim3(threads), 0, st, a);
  else if (its == 2) launch_pdl(stream_norm_kernel<A, S, 2>, dim3(T), dim3(threads), 0, st, a);
  else if (its <= 4) launch_pdl(stream_norm_kernel<A, S, 4>, dim3(T), dim3(threads), 0, st, a);
  else if (its <= 8) launch_pdl(stream_norm_kernel<A, S, 8>, dim3(T), dim3(threads), 0, st, a);
  else {
    const size_t smem = static_cast<size_t>(a.W) * sizeof(float);
    if (smem > 40 * 1024 &&
        cudaFuncSetAttribute(stream_norm_kernel<A, S, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
      return -3;
    launch_pdl(stream_norm_kernel<A, S, 0>, dim3(T), dim3(threads), smem, st, a);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <typename A>
static int launch_streams(const StreamArgs<A>& a, int S, int T, cudaStream_t st) {
  switch (S) {
    case 1: return launch_stream_norm<A, 1>(a, T, st);
    case 2: return launch_stream_norm<A, 2>(a, T, st);
    case 3: return launch_stream_norm<A, 3>(a, T, st);
    case 4: return launch_stream_norm<A, 4>(a, T, st);
    case 5: return launch_stream_norm<A, 5>(a, T, st);
    case 6: return launch_stream_norm<A, 6>(a, T, st);
    case 7: return launch_stream_norm<A, 7>(a, T, st);
    default: return launch_stream_norm<A, 8>(a, T, st);
  }
}

// out[t, mix : o0) = 0, out[t, o0 + j] = act(gate_j) * up_j for j < ff, zero up to `cols`.  relu: act is relu, else silu.
template <typename A>
__global__ void __launch_bounds__(256)
join_glu_kernel(const A* __restrict__ proj, long long ldp, int go, int uo, int ff, A* __restrict__ out, long long ldo, int mix,
                int o0, int cols, int relu) {
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.y;
  const A* pg = proj + t * ldp + go;
  const A* pu = proj + t * ldp + uo;
  A* o = out + t * ldo;
  const int base = blockIdx.x * blockDim.x * 8 + threadIdx.x * 8;      // eight columns per thread, from o0 on
  if (blockIdx.x == 0)
    for (int i = mix + threadIdx.x; i < o0; i += blockDim.x) st_act(o + i, 0.f);
  glu_columns(pg, pu, o + o0, base, ff, cols - o0, (ldo & 7) == 0 && (ldp & 7) == 0, relu);
}

// out[t, c] = xIELU(z[t, c]) = (z > 0 ? a z^2 : b (exp(z) - 1 - z)) + z / 2 for c < ff, zero up to `width`; eight columns per thread.
template <typename A>
__global__ void __launch_bounds__(256)
xielu_kernel(const A* __restrict__ z, long long ldz, int ff, float a, float b, A* __restrict__ out, long long ldo, int width, int T) {
  pdl_wait();
  pdl_trigger();
  const int c0 = (blockIdx.y * 256 + threadIdx.x) * 8;
  if (c0 >= width) return;
  const long long t = blockIdx.x;
  auto f = [&](float x) {
    if (sizeof(A) == 4) return fmaf(x, 0.5f, x > 0.f ? a * x * x : b * (expm1f(x) - x));
    // rounded results: exp(x) - 1 - x from its series where the difference would cancel
    const float near = x * x * fmaf(x, fmaf(x, fmaf(x, 1.f / 120.f, 1.f / 24.f), 1.f / 6.f), 0.5f), far = __expf(x) - 1.f - x;
    return fmaf(x, 0.5f, x > 0.f ? a * x * x : b * (x > -0.25f ? near : far));
  };
  const A* p = z + t * ldz + c0;
  A* o = out + t * ldo + c0;
  if (sizeof(A) == 2 && c0 + 8 <= ff && ((ldz | ldo) & 7) == 0) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    uint4 r;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 x = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&v)[j]);
      // two at a time: the series and the difference of f in packed arithmetic
      const uint64_t xx = pack2(x.x, x.y), sq = mul2(xx, xx);
      const uint64_t near = mul2(sq, fma2(xx, fma2(xx, fma2(xx, pack2(1.f / 120.f, 1.f / 120.f), pack2(1.f / 24.f, 1.f / 24.f)),
                                                   pack2(1.f / 6.f, 1.f / 6.f)), pack2(0.5f, 0.5f)));
      float n0, n1, q0, q1, y0, y1;
      unpack2(near, n0, n1);
      unpack2(sq, q0, q1);
      const float e0 = __expf(x.x) - 1.f - x.x, e1 = __expf(x.y) - 1.f - x.y;
      const uint64_t by = pack2(x.x > 0.f ? a : b, x.y > 0.f ? a : b);
      const uint64_t part = pack2(x.x > 0.f ? q0 : x.x > -0.25f ? n0 : e0, x.y > 0.f ? q1 : x.y > -0.25f ? n1 : e1);
      unpack2(fma2(part, by, mul2(xx, pack2(0.5f, 0.5f))), y0, y1);
      reinterpret_cast<__nv_bfloat162*>(&r)[j] = __floats2bfloat162_rn(y0, y1);
    }
    *reinterpret_cast<uint4*>(o) = r;
    return;
  }
  for (int j = 0; j < 8 && c0 + j < width; ++j) st_act(o + j, c0 + j < ff ? f(ld_act(p + j)) : 0.f);
}

}  // namespace stk

using namespace stk;

// z and out rows start on 16 bytes.
STK_API int stk_xielu(const void* z, long long ldz, int ff, float a, float b, void* out, long long ldo, int width, int fp32, int T,
                      void* stream) {
  if (T <= 0) return 0;
  if (width < ff || ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 15)) return -1;
  const dim3 grid(static_cast<unsigned>(T), static_cast<unsigned>((width + 2047) / 2048));
  cudaStream_t st = (cudaStream_t)stream;
  if (fp32) launch_pdl(xielu_kernel<float>, grid, dim3(256), 0, st, (const float*)z, ldz, ff, a, b, (float*)out, ldo, width, T);
  else launch_pdl(xielu_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, (const __nv_bfloat16*)z, ldz, ff, a, b, (__nv_bfloat16*)out, ldo, width, T);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_embed_scaled(const int64_t* ids, const void* embed, int embed_fp32, float* x, long long ldx, int copies, int T, int W,
                             int vocab, float scale, void* h, long long ldh, int width, int* status, void* stream) {
  if (T <= 0) return 0;
  cudaStream_t st = (cudaStream_t)stream;
  if (embed_fp32)
    launch_pdl(embed_scaled_kernel<float>, dim3(T), dim3(256), 0, st, ids, (const float*)embed, x, ldx, copies, W, vocab, scale, (float*)h,
               ldh, width, status);
  else
    launch_pdl(embed_scaled_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, st, ids, (const __nv_bfloat16*)embed, x, ldx, copies, W, vocab,
               scale, (__nv_bfloat16*)h, ldh, width, status);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_add_layer_norm(float* x, long long ldx, const float* y, long long ldy, const float* w, void* h, int h_fp32,
                               long long ldh, int T, int W, int width, float eps, const int64_t* rows, int center, void* stream) {
  if (T <= 0) return 0;
  const size_t smem = static_cast<size_t>(W) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  if (smem > 40 * 1024) {
    if (cudaFuncSetAttribute(add_layer_norm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) !=
            cudaSuccess ||
        cudaFuncSetAttribute(add_layer_norm_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) !=
            cudaSuccess)
      return -3;
  }
  // few rows: a wide row is spread over more threads (the step waits for this kernel); many rows: more rows at once
  const int threads = T > 148 || W <= 1024 ? 256 : (W <= 2048 ? 512 : 1024);
  if (h_fp32)
    launch_pdl(add_layer_norm_kernel<float>, dim3(T), dim3(threads), smem, st, x, ldx, y, ldy, w, (float*)h, ldh, W, width, eps, rows,
               center);
  else
    launch_pdl(add_layer_norm_kernel<__nv_bfloat16>, dim3(T), dim3(threads), smem, st, x, ldx, y, ldy, w, (__nv_bfloat16*)h, ldh, W,
               width, eps, rows, center);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

STK_API int stk_join_glu(const void* proj, long long ldp, int gate_off, int up_off, int ff, void* out, long long ldo, int fp32,
                         int mixer_dim, int ff_off, int cols, int relu, int T, void* stream) {
  if (T <= 0) return 0;
  if (T > 65535) return -1;
  const int n = cols - ff_off;
  const dim3 grid(n > 0 ? (n + 2047) / 2048 : 1, T);
  cudaStream_t st = (cudaStream_t)stream;
  if (fp32)
    launch_pdl(join_glu_kernel<float>, grid, dim3(256), 0, st, (const float*)proj, ldp, gate_off, up_off, ff, (float*)out, ldo,
               mixer_dim, ff_off, cols, relu);
  else
    launch_pdl(join_glu_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, (const __nv_bfloat16*)proj, ldp, gate_off, up_off, ff,
               (__nv_bfloat16*)out, ldo, mixer_dim, ff_off, cols, relu);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// pairs == nullptr: y [T, W] fp32 rows.  Otherwise the weighted sum of each token's `top` expert rows in the compute type.
STK_API int stk_post_norm_add(float* x, long long ldx, const float* y, long long ldy, const void* pairs, long long ldp,
                              const int* pair_row, const float* weights, int top, const float* w, float eps, void* h, long long ldh,
                              int W, int width, int fp32, int T, void* stream) {
  if (T <= 0) return 0;
  const size_t smem = static_cast<size_t>(W) * sizeof(float);
  if (smem > 200 * 1024 || top > 32 || (pairs == nullptr) == (y == nullptr)) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  if (smem > 40 * 1024) {
    if (cudaFuncSetAttribute(post_norm_add_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess ||
        cudaFuncSetAttribute(post_norm_add_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) !=
            cudaSuccess)
      return -3;
  }
  const int threads = T > 148 || W <= 1024 ? 256 : (W <= 2048 ? 512 : 1024);
  if (fp32) {
    const PostNormArgs<float> a{x, ldx, y, ldy, (const float*)pairs, ldp, pair_row, weights, top, w, eps, (float*)h, ldh, W, width};
    launch_pdl(post_norm_add_kernel<float>, dim3(T), dim3(threads), smem, st, a);
  } else {
    const PostNormArgs<__nv_bfloat16> a{x,   ldx, y, ldy, (const __nv_bfloat16*)pairs, ldp, pair_row, weights, top,
                                        w, eps, (__nv_bfloat16*)h, ldh, W, width};
    launch_pdl(post_norm_add_kernel<__nv_bfloat16>, dim3(T), dim3(threads), smem, st, a);
  }
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// x [*, streams, W].  pairs == nullptr: y [*, W] fp32 rows (neither: the streams stay as they are).  mix [streams, streams] indexed
// [from, to], write and read [streams].  T rows are normed: all, or those in `rows`.
STK_API int stk_stream_norm(float* x, int streams, const float* y, long long ldy, const void* pairs, long long ldp, const int* pair_row,
                            const float* weights, int top, const float* mix, const float* write, const float* read, const float* w,
                            const float* b, float eps, void* h, long long ldh, int W, int width, int fp32, const int64_t* rows, int T,
                            void* stream) {
  if (T <= 0) return 0;
  if (streams < 1 || streams > 8 || static_cast<size_t>(W) * sizeof(float) > 200 * 1024 || top > 32 ||
      (pairs != nullptr && y != nullptr))
    return -2;
  cudaStream_t st = (cudaStream_t)stream;
  if (fp32) {
    const StreamArgs<float> a{x, y, ldy, (const float*)pairs, ldp, pair_row, weights, top, mix, write, read, w, b, eps, (float*)h, ldh,
                              W, width, rows};
    return launch_streams(a, streams, T, st);
  }
  const StreamArgs<__nv_bfloat16> a{x, y, ldy, (const __nv_bfloat16*)pairs, ldp, pair_row, weights, top, mix, write, read, w, b, eps,
                                    (__nv_bfloat16*)h, ldh, W, width, rows};
  return launch_streams(a, streams, T, st);
}
