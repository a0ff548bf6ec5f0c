// What a token takes from the one before it (ops/shifted.py): the bigram embedding, and the shifted norm of "shifted" blocks.
//
//   embed_bigram      x = embed[token] * scale + table[(previous * mul_prev + token * mul_cur) mod buckets]
//   shifted_norm      x += what the layer before left;  h = rms_norm(x);  s = h + (h' - h) shift;  blend_j = s + (s' - s) mu_j, where h'
//                     and s' are the previous token's h and s
//   shift_commit      the last h, s and token of every request's span become its state
//
//   sum_norm          x and h alone: the model's last norm, and the first half of long steps
//   shift_blend       s and the blends of long steps, from x and 1 / rms
//
// shifted_norm: a CTA walks a run of consecutive tokens with h' and s' in registers.  At the start of a run it forms h of the two tokens
// before it once more (s' needs the h before that), at the start of a span it takes h' and s' from the request's state.  The new
// state goes to a second buffer: other CTAs of the step may still read the first.
#define STK_PDL_CLASS 4
#include "hybrid_block.cuh"

namespace stk {

template <typename E>
__global__ void __launch_bounds__(256)
embed_bigram_kernel(const int64_t* __restrict__ ids, const E* __restrict__ embed, float scale, const E* __restrict__ table, long long buckets,
                    long long mul_prev, long long mul_cur, const int* __restrict__ tok_req, const int64_t* __restrict__ positions,
                    const int* __restrict__ first_pos, const int64_t* __restrict__ last_token, float* __restrict__ x, int W, int vocab,
                    int* status) {
  pdl_wait();
  pdl_trigger();
  const int t = blockIdx.x;
  const long long id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0) set_status(status, kBadIndex, t);
  const int req = tok_req[t];
  const long long pos = positions[t];
  long long row = -1;
  if (table != nullptr && ok && req >= 0 && pos >= 0) {
    row = buckets;
    if (pos > 0) {
      const long long prev = pos > first_pos[t] ? ids[t - 1] : last_token[req];
      row = (prev * mul_prev + id * mul_cur) % buckets;
      if (row < 0) row = -1;                               // a previous token that does not exist: reported where it was read
    }
  }
  float* to = x + static_cast<long long>(t) * W;
  if (sizeof(E) == 2 && (W & 7) == 0) {
    for (int i = threadIdx.x * 8; i < W; i += blockDim.x * 8) {
      uint4 a = make_uint4(0, 0, 0, 0), b = a;
      if (ok) a = __ldg(reinterpret_cast<const uint4*>(embed + id * W + i));
      if (row >= 0) b = __ldg(reinterpret_cast<const uint4*>(table + row * W + i));
      float f[8];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 u = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&a)[j]);
        const float2 v = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&b)[j]);
        f[2 * j] = fmaf(u.x, scale, v.x);
        f[2 * j + 1] = fmaf(u.y, scale, v.y);
      }
      *reinterpret_cast<float4*>(to + i) = make_float4(f[0], f[1], f[2], f[3]);
      *reinterpret_cast<float4*>(to + i + 4) = make_float4(f[4], f[5], f[6], f[7]);
    }
    return;
  }
  for (int i = threadIdx.x; i < W; i += blockDim.x)
    to[i] = fmaf(ok ? ld_act(embed + id * W + i) : 0.f, scale, row >= 0 ? ld_act(table + row * W + i) : 0.f);
}

struct ShiftOut { const float* y; long long ld; const float* w; float f; };      // f * rms_norm(y) * w (w null: f * y)

template <typename A>
struct ShiftArgs {
  const float* x; float* x_out;
  ShiftOut o[2];
  const float* ff; long long ldf;
  const A* pairs; long long ldp; const int* pair_row; const float* weights; int top;
  const float* norm; float eps;
  const float* shift; const float* mu; int blends;
  A* h; A* s; A* mix;
  const float* now; float* then;                  // [rows][2][W]
  const int* tok_req; const int64_t* positions; const int* first_pos; const int* last_pos;
  const int64_t* rows;
  int T, W, width, run;
  float* inv;                                     // [T] receives 1 / rms(x) (or null)
};

// N columns (4, or 1 for widths that are not multiples of 4) from p.
template <int N>
__device__ __forceinline__ void sh_load(const float* p, float (&v)[N]) {
  if constexpr (N == 4) {
    const float4 f = *reinterpret_cast<const float4*>(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    v[0] = *p;
  }
}
template <int N>
__device__ __forceinline__ void sh_store(float* p, const float (&v)[N]) {
  if constexpr (N == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else *p = v[0];
}
template <typename A, int N>
__device__ __forceinline__ void sh_store_act(A* p, const float (&v)[N]) {
  if constexpr (N == 4 && sizeof(A) == 2) {
    __align__(8) const __nv_bfloat162 b[2] = {__floats2bfloat162_rn(v[0], v[1]), __floats2bfloat162_rn(v[2], v[3])};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(b);
  } else if constexpr (N == 4) {
    sh_store<4>(reinterpret_cast<float*>(p), v);
  } else {
    st_act(p, v[0]);
  }
}
// Two block-wide sums at once (red: 64 floats).
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  __syncthreads();
  if (lane == 0) { red[warp] = a; red[32 + warp] = b; }
  __syncthreads();
  a = lane < nw ? red[lane] : 0.f;
  b = lane < nw ? red[32 + lane] : 0.f;
  return make_float2(warp_sum(a), warp_sum(b));
}

// v += N columns of the feed-forward's output: a row, or the weighted sum of a token's expert rows.
template <typename A, int N>
__device__ __forceinline__ void sh_tail(const ShiftArgs<A>& a, long long r, int i, const long long* src, const float* wt, float (&v)[N]) {
  if (a.ff != nullptr) {
    float f[N];
    sh_load<N>(a.ff + r * a.ldf + i, f);
#pragma unroll
    for (int k = 0; k < N; ++k) v[k] += f[k];
  }
  if (a.pairs != nullptr) {
    float f[N];
#pragma unroll
    for (int k = 0; k < N; ++k) f[k] = 0.f;
    if constexpr (N == 4 && sizeof(A) == 2) {
      for (int j0 = 0; j0 < a.top; j0 += 4) {                 // four rows in flight
        uint2 q[4];
#pragma unroll
        for (int j = 0; j < 4; ++j)
          q[j] = j0 + j < a.top ? *reinterpret_cast<const uint2*>(a.pairs + src[j0 + j] + i) : make_uint2(0, 0);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float w = j0 + j < a.top ? wt[j0 + j] : 0.f;
          const float2 f0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q[j].x));
          const float2 f1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q[j].y));
          f[0] = fmaf(w, f0.x, f[0]); f[1] = fmaf(w, f0.y, f[1]);
          f[2] = fmaf(w, f1.x, f[2]); f[3] = fmaf(w, f1.y, f[3]);
        }
      }
    } else {
      for (int j = 0; j < a.top; ++j)
#pragma unroll
        for (int k = 0; k < N; ++k) f[k] = fmaf(wt[j], ld_act(a.pairs + src[j] + i + k), f[k]);
    }
#pragma unroll
    for (int k = 0; k < N; ++k) v[k] += f[k];
  }
}

__device__ __forceinline__ void sh_prefetch(const float* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }

template <typename A, int N, int NIT, int THREADS>
__global__ void __launch_bounds__(THREADS)
shifted_norm_kernel(const ShiftArgs<A> a) {
  __shared__ float red[64], red1[32];
  __shared__ long long src[32];
  __shared__ float wt[32];
  constexpr int kMu = NIT > 1 ? 0 : THREADS > 256 ? 2 : 5;                // blends whose weights are asked for before the last wait
  if (blockIdx.x == 0) {
    // the weights come from HBM while the kernel before is at work
    for (int i = threadIdx.x * 32; i < a.W; i += blockDim.x * 32) {
      if (a.o[0].w != nullptr) sh_prefetch(a.o[0].w + i);
      if (a.o[1].w != nullptr) sh_prefetch(a.o[1].w + i);
      sh_prefetch(a.norm + i);
      sh_prefetch(a.shift + i);
      for (int j = 0; j < a.blends; ++j) sh_prefetch(a.mu + static_cast<long long>(j) * a.W + i);
    }
  }
  pdl_wait();
  pdl_trigger();
  const int step = blockDim.x * N, i0 = threadIdx.x * N;
  const int r0 = blockIdx.x * a.run, r1 = min(a.T, r0 + a.run);
  const float inv_w = 1.f / static_cast<float>(a.W);
  int begin = r0;
  if (a.run > 1 && a.tok_req[r0] >= 0 && a.positions[r0] >= 0)
    begin = r0 - static_cast<int>(min(2ll, static_cast<long long>(a.positions[r0]) - a.first_pos[r0]));
  float hp[NIT][N], sp[NIT][N];
#pragma unroll
  for (int e = 0; e < NIT; ++e)
#pragma unroll
    for (int k = 0; k < N; ++k) hp[e][k] = sp[e][k] = 0.f;
  for (int t = begin; t < r1; ++t) {
    const bool own = t >= r0;
    const long long r = t;
    const int req = a.tok_req[t];
    const long long pos = a.positions[t];
    if (req >= 0 && pos == a.first_pos[t]) {
      const float* st = a.now + static_cast<long long>(req) * 2 * a.W;
#pragma unroll
      for (int e = 0; e < NIT; ++e) {
        const int i = i0 + e * step;
        if (pos > 0 && i < a.W) {
          sh_load<N>(st + i, hp[e]);
          sh_load<N>(st + a.W + i, sp[e]);
        } else {
#pragma unroll
          for (int k = 0; k < N; ++k) hp[e][k] = sp[e][k] = 0.f;
        }
      }
    }
    if (a.pairs != nullptr) {
      __syncthreads();
      if (static_cast<int>(threadIdx.x) < a.top) {
        const long long p = r * a.top + threadIdx.x;
        const int at = a.pair_row != nullptr ? a.pair_row[p] : static_cast<int>(p);
        src[threadIdx.x] = at < 0 ? 0 : at * a.ldp;
        wt[threadIdx.x] = at < 0 ? 0.f : a.weights[p];
      }
      __syncthreads();
    }
    float v[NIT][N], y0[NIT][N], y1[NIT][N], q0 = 0.f, q1 = 0.f;
#pragma unroll
    for (int e = 0; e < NIT; ++e) {
      const int i = i0 + e * step;
#pragma unroll
      for (int k = 0; k < N; ++k) v[e][k] = y0[e][k] = y1[e][k] = 0.f;
      if (i >= a.W) continue;
      sh_load<N>(a.x + r * a.W + i, v[e]);
      if (a.o[0].y != nullptr) sh_load<N>(a.o[0].y + r * a.o[0].ld + i, y0[e]);
      if (a.o[1].y != nullptr) sh_load<N>(a.o[1].y + r * a.o[1].ld + i, y1[e]);
      sh_tail<A, N>(a, r, i, src, wt, v[e]);
#pragma unroll
      for (int k = 0; k < N; ++k) {
        q0 = fmaf(y0[e][k], y0[e][k], q0);
        q1 = fmaf(y1[e][k], y1[e][k], q1);
      }
    }
    float f0 = a.o[0].f, f1 = a.o[1].f;
    float u0[NIT][N], u1[NIT][N];                                       // the outputs' weights, before the wait as well
#pragma unroll
    for (int e = 0; e < NIT; ++e) {
      const int i = i0 + e * step;
      if (NIT > 1 || i >= a.W) continue;
      if (a.o[0].w != nullptr) sh_load<N>(a.o[0].w + i, u0[e]);
      if (a.o[1].w != nullptr) sh_load<N>(a.o[1].w + i, u1[e]);
    }
    if (a.o[0].w != nullptr || a.o[1].w != nullptr) {
      const float2 q = block_sum2(q0, q1, red);
      if (a.o[0].w != nullptr) f0 /= sqrtf(q.x * inv_w + a.eps);
      if (a.o[1].w != nullptr) f1 /= sqrtf(q.y * inv_w + a.eps);
    }
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < NIT; ++e) {
      const int i = i0 + e * step;
      if (i >= a.W) continue;
      if (a.o[0].y != nullptr) {
        if (NIT > 1 && a.o[0].w != nullptr) sh_load<N>(a.o[0].w + i, u0[e]);
#pragma unroll
        for (int k = 0; k < N; ++k) v[e][k] = fmaf(y0[e][k] * f0, a.o[0].w != nullptr ? u0[e][k] : 1.f, v[e][k]);
      }
      if (a.o[1].y != nullptr) {
        if (NIT > 1 && a.o[1].w != nullptr) sh_load<N>(a.o[1].w + i, u1[e]);
#pragma unroll
        for (int k = 0; k < N; ++k) v[e][k] = fmaf(y1[e][k] * f1, a.o[1].w != nullptr ? u1[e][k] : 1.f, v[e][k]);
      }
      if (own && a.x_out != nullptr) sh_store<N>(a.x_out + r * a.W + i, v[e]);
#pragma unroll
      for (int k = 0; k < N; ++k) ss = fmaf(v[e][k], v[e][k], ss);
    }
    // what the rest needs is asked for before the wait
    float wn[NIT][N], ws[NIT][N], wm[kMu > 0 ? kMu : 1][N];
#pragma unroll
    for (int e = 0; e < NIT; ++e) {
      const int i = i0 + e * step;
      if (NIT > 1 || i >= a.W) continue;
#pragma unroll
      for (int j = 0; j < kMu; ++j)
        if (j < a.blends) sh_load<N>(a.mu + static_cast<long long>(j) * a.W + i, wm[j]);
      sh_load<N>(a.norm + i, wn[e]);
      sh_load<N>(a.shift + i, ws[e]);
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red1) * inv_w + a.eps);
    const bool keep = own && req >= 0 && pos == a.last_pos[t];
    float* st = keep ? a.then + static_cast<long long>(req) * 2 * a.W : nullptr;
#pragma unroll
    for (int e = 0; e < NIT; ++e) {
      const int i = i0 + e * step;
      if (i >= a.W) continue;
      float w[N], h[N], s[N];
      if (NIT > 1) sh_load<N>(a.norm + i, wn[e]);
#pragma unroll
      for (int k = 0; k < N; ++k) h[k] = v[e][k] * inv * wn[e][k];
      if (own) sh_store_act<A, N>(a.h + static_cast<long long>(t) * a.width + i, h);
      if (NIT > 1) sh_load<N>(a.shift + i, ws[e]);
#pragma unroll
      for (int k = 0; k < N; ++k) s[k] = fmaf(hp[e][k] - h[k], ws[e][k], h[k]);
      if (own) {
        sh_store_act<A, N>(a.s + static_cast<long long>(t) * a.width + i, s);
        auto blend = [&](int j, const float (&m)[N]) {
          float b[N];
#pragma unroll
          for (int k = 0; k < N; ++k) b[k] = fmaf(sp[e][k] - s[k], m[k], s[k]);
          sh_store_act<A, N>(a.mix + (static_cast<long long>(t) * a.blends + j) * a.width + i, b);
        };
#pragma unroll
        for (int j = 0; j < kMu; ++j)
          if (j < a.blends) blend(j, wm[j]);
        for (int j = kMu; j < a.blends; ++j) {
          sh_load<N>(a.mu + static_cast<long long>(j) * a.W + i, w);
          blend(j, w);
        }
        if (keep) {
          sh_store<N>(st + i, h);
          sh_store<N>(st + a.W + i, s);
        }
      }
#pragma unroll
      for (int k = 0; k < N; ++k) { hp[e][k] = h[k]; sp[e][k] = s[k]; }
    }
    if (own)
      for (int i = a.W + threadIdx.x; i < a.width; i += blockDim.x) {
        st_act(a.h + static_cast<long long>(t) * a.width + i, 0.f);
        st_act(a.s + static_cast<long long>(t) * a.width + i, 0.f);
        for (int j = 0; j < a.blends; ++j) st_act(a.mix + (static_cast<long long>(t) * a.blends + j) * a.width + i, 0.f);
      }
  }
}

// The sum and the norm alone: the first half of a long step, and the model's last norm (rows: only of these tokens, the sum is not kept).
template <typename A, int N, int NIT, int THREADS>
__global__ void __launch_bounds__(THREADS, 1024 / THREADS)
sum_norm_kernel(const ShiftArgs<A> a) {
  __shared__ float red[64], red1[32];
  __shared__ long long src[32];
  __shared__ float wt[32];
  pdl_wait();
  pdl_trigger();
  const int step = blockDim.x * N, i0 = threadIdx.x * N;
  const float inv_w = 1.f / static_cast<float>(a.W);
  const long long r = a.rows != nullptr ? a.rows[blockIdx.x] : static_cast<long long>(blockIdx.x);
  if (a.pairs != nullptr && static_cast<int>(threadIdx.x) < a.top) {
    const long long p = r * a.top + threadIdx.x;
    const int at = a.pair_row != nullptr ? a.pair_row[p] : static_cast<int>(p);
    src[threadIdx.x] = at < 0 ? 0 : at * a.ldp;
    wt[threadIdx.x] = at < 0 ? 0.f : a.weights[p];
  }
  float v[NIT][N], y0[NIT][N], y1[NIT][N], q0 = 0.f, q1 = 0.f;
#pragma unroll
  for (int e = 0; e < NIT; ++e) {
    const int i = i0 + e * step;
#pragma unroll
    for (int k = 0; k < N; ++k) v[e][k] = y0[e][k] = y1[e][k] = 0.f;
    if (i >= a.W) continue;
    sh_load<N>(a.x + r * a.W + i, v[e]);
    if (a.o[0].y != nullptr) sh_load<N>(a.o[0].y + r * a.o[0].ld + i, y0[e]);
    if (a.o[1].y != nullptr) sh_load<N>(a.o[1].y + r * a.o[1].ld + i, y1[e]);
  }
  if (a.pairs != nullptr) __syncthreads();
#pragma unroll
  for (int e = 0; e < NIT; ++e) {
    const int i = i0 + e * step;
    if (i >= a.W) continue;
    sh_tail<A, N>(a, r, i, src, wt, v[e]);
#pragma unroll
    for (int k = 0; k < N; ++k) {
      q0 = fmaf(y0[e][k], y0[e][k], q0);
      q1 = fmaf(y1[e][k], y1[e][k], q1);
    }
  }
  float f0 = a.o[0].f, f1 = a.o[1].f;
  if (a.o[0].w != nullptr || a.o[1].w != nullptr) {
    const float2 q = block_sum2(q0, q1, red);
    if (a.o[0].w != nullptr) f0 /= sqrtf(q.x * inv_w + a.eps);
    if (a.o[1].w != nullptr) f1 /= sqrtf(q.y * inv_w + a.eps);
  }
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < NIT; ++e) {
    const int i = i0 + e * step;
    if (i >= a.W) continue;
    float u0[N], u1[N];
    if (a.o[0].w != nullptr) sh_load<N>(a.o[0].w + i, u0);
    if (a.o[1].w != nullptr) sh_load<N>(a.o[1].w + i, u1);
#pragma unroll
    for (int k = 0; k < N; ++k) {
      if (a.o[0].y != nullptr) v[e][k] = fmaf(y0[e][k] * f0, a.o[0].w != nullptr ? u0[k] : 1.f, v[e][k]);
      if (a.o[1].y != nullptr) v[e][k] = fmaf(y1[e][k] * f1, a.o[1].w != nullptr ? u1[k] : 1.f, v[e][k]);
      ss = fmaf(v[e][k], v[e][k], ss);
    }
    if (a.x_out != nullptr) sh_store<N>(a.x_out + r * a.W + i, v[e]);
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red1) * inv_w + a.eps);
  if (a.inv != nullptr && threadIdx.x == 0) a.inv[blockIdx.x] = inv;
  A* to = a.h + static_cast<long long>(blockIdx.x) * a.width;
#pragma unroll
  for (int e = 0; e < NIT; ++e) {
    const int i = i0 + e * step;
    if (i >= a.W) continue;
    float w[N], h[N];
    sh_load<N>(a.norm + i, w);
#pragma unroll
    for (int k = 0; k < N; ++k) h[k] = v[e][k] * inv * w[k];
    sh_store_act<A, N>(to + i, h);
  }
  for (int i = a.W + threadIdx.x; i < a.width; i += blockDim.x) st_act(to + i, 0.f);
}

// The second half of a long step: shifted rows and blends of N columns per thread over a run of tokens.  h is formed again from the residual and
// 1 / rms, in fp32.
template <typename A>
struct BlendArgs {
  const float* x; const float* inv;
  const float* norm; const float* shift; const float* mu;
  A* s; A* mix;
  const float* now; float* then;
  const int* tok_req; const int64_t* positions; const int* first_pos; const int* last_pos;
  int T, W, width;
};
constexpr int kBlendRun = 16, kBlendAhead = 4;

template <typename A, int N, int BLENDS>
__global__ void __launch_bounds__(256, 4)
shift_blend_kernel(const BlendArgs<A> a) {
  __shared__ __align__(16) float wts[2 + BLENDS][256 * N];        // norm, shift, mu of the thread's columns
  __shared__ float s_inv[kBlendRun + 2];
  __shared__ int s_req[kBlendRun + 2], s_kind[kBlendRun + 2];     // kind: 1 first of its span with a state, 2 first without, 4 last
  pdl_wait();
  pdl_trigger();
  const int i = (blockIdx.x * blockDim.x + threadIdx.x) * N, at = threadIdx.x * N;
  const int r0 = blockIdx.y * kBlendRun, r1 = min(a.T, r0 + kBlendRun);
  int begin = r0;
  if (a.tok_req[r0] >= 0 && a.positions[r0] >= 0)
    begin = r0 - static_cast<int>(min(2ll, static_cast<long long>(a.positions[r0]) - a.first_pos[r0]));
  if (static_cast<int>(threadIdx.x) < r1 - begin) {
    const int t = begin + threadIdx.x, req = a.tok_req[t];
    const long long pos = a.positions[t];
    s_inv[threadIdx.x] = a.inv[t];
    s_req[threadIdx.x] = req;
    s_kind[threadIdx.x] = req < 0 ? 0 : (pos == a.first_pos[t] ? (pos > 0 ? 1 : 2) : 0) | (pos == a.last_pos[t] ? 4 : 0);
  }
  const bool in = i < a.W;
  if (in) {
    float w[N];
    sh_load<N>(a.norm + i, w);
    sh_store<N>(&wts[0][at], w);
    sh_load<N>(a.shift + i, w);
    sh_store<N>(&wts[1][at], w);
#pragma unroll
    for (int j = 0; j < BLENDS; ++j) {
      sh_load<N>(a.mu + static_cast<long long>(j) * a.W + i, w);
      sh_store<N>(&wts[2 + j][at], w);
    }
  }
  __syncthreads();
  if (!in) {
    // zeros behind the last column
    for (int t = r0; i < a.width && t < r1; ++t)
      for (int k = 0; k < N && i + k < a.width; ++k) {
        st_act(a.s + static_cast<long long>(t) * a.width + i + k, 0.f);
        for (int j = 0; j < BLENDS; ++j) st_act(a.mix + (static_cast<long long>(t) * BLENDS + j) * a.width + i + k, 0.f);
      }
    return;
  }
  float hp[N], sp[N], x[kBlendAhead][N];
#pragma unroll
  for (int k = 0; k < N; ++k) hp[k] = sp[k] = 0.f;
#pragma unroll
  for (int j = 0; j < kBlendAhead; ++j)
    if (begin + j < r1) sh_load<N>(a.x + (begin + static_cast<long long>(j)) * a.W + i, x[j]);
  for (int t0 = begin; t0 < r1; t0 += kBlendAhead) {
#pragma unroll
    for (int u = 0; u < kBlendAhead; ++u) {
      const int t = t0 + u;
      if (t >= r1) break;
      const float inv = s_inv[t - begin];
      const int kind = s_kind[t - begin];
      float h[N], s[N], w[N];
      sh_load<N>(&wts[0][at], w);
#pragma unroll
      for (int k = 0; k < N; ++k) h[k] = x[u][k] * inv * w[k];
      if (t + kBlendAhead < r1) sh_load<N>(a.x + (t + static_cast<long long>(kBlendAhead)) * a.W + i, x[u]);
      if (kind & 3) {
        if (kind & 1) {
          const float* st = a.now + static_cast<long long>(s_req[t - begin]) * 2 * a.W;
          sh_load<N>(st + i, hp);
          sh_load<N>(st + a.W + i, sp);
        } else {
#pragma unroll
          for (int k = 0; k < N; ++k) hp[k] = sp[k] = 0.f;
        }
      }
      sh_load<N>(&wts[1][at], w);
#pragma unroll
      for (int k = 0; k < N; ++k) s[k] = fmaf(hp[k] - h[k], w[k], h[k]);
      if (t >= r0) {
        sh_store_act<A, N>(a.s + static_cast<long long>(t) * a.width + i, s);
#pragma unroll
        for (int j = 0; j < BLENDS; ++j) {
          float b[N];
          sh_load<N>(&wts[2 + j][at], w);
#pragma unroll
          for (int k = 0; k < N; ++k) b[k] = fmaf(sp[k] - s[k], w[k], s[k]);
          sh_store_act<A, N>(a.mix + (static_cast<long long>(t) * BLENDS + j) * a.width + i, b);
        }
        if (kind & 4) {
          float* st = a.then + static_cast<long long>(s_req[t - begin]) * 2 * a.W;
          sh_store<N>(st + i, h);
          sh_store<N>(st + a.W + i, s);
        }
      }
#pragma unroll
      for (int k = 0; k < N; ++k) { hp[k] = h[k]; sp[k] = s[k]; }
    }
  }
}


template <typename A>
static int launch_sum_norm(const ShiftArgs<A>& a, bool vec, cudaStream_t st) {
  const int need = (a.W + (vec ? 4 : 1) - 1) / (vec ? 4 : 1);
  // many tokens: two groups of columns per thread keep enough loads in flight; few: a wide row is spread over more threads
  const int threads = need <= 256 ? 256 : a.T > 148 ? (need <= 512 ? 256 : need <= 1024 ? 512 : 1024) : need <= 512 ? 512 : 1024;
  const int its = (need + threads - 1) / threads;
#define STK_SUM(N, NIT)                                                                                              \
  do {                                                                                                               \
    if (threads == 256) launch_pdl(sum_norm_kernel<A, N, NIT, 256>, dim3(a.T), dim3(256), 0, st, a);                 \
    else if (threads == 512) launch_pdl(sum_norm_kernel<A, N, NIT, 512>, dim3(a.T), dim3(512), 0, st, a);            \
    else launch_pdl(sum_norm_kernel<A, N, NIT, 1024>, dim3(a.T), dim3(1024), 0, st, a);                              \
  } while (0)
  if (vec) {
    if (its == 1) STK_SUM(4, 1);
    else if (its == 2) STK_SUM(4, 2);
    else if (its <= 4) STK_SUM(4, 4);
    else return -2;
  } else {
    if (its == 1) STK_SUM(1, 1);
    else if (its <= 4) STK_SUM(1, 4);
    else if (its <= 16) STK_SUM(1, 16);
    else return -2;
  }
#undef STK_SUM
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

template <typename A>
static int launch_shifted(ShiftArgs<A> a, float* inv, int decode, int sm_count, cudaStream_t st) {
  const bool vec = a.W % 4 == 0 && a.o[0].ld % 4 == 0 && a.o[1].ld % 4 == 0 && a.ldf % 4 == 0 && a.ldp % 4 == 0 && a.width % 4 == 0;
  if (a.shift == nullptr) return launch_sum_norm(a, vec, st);
  if (!decode && inv != nullptr && a.T > 2 * sm_count && (a.blends == 0 || a.blends == 5)) {
    ShiftArgs<A> sum = a;
    sum.inv = inv;
    const int rc = launch_sum_norm(sum, vec, st);
    if (rc != 0) return rc;
    const BlendArgs<A> b{a.x_out != nullptr ? a.x_out : a.x, inv, a.norm, a.shift, a.mu, a.s, a.mix, a.now, a.then, a.tok_req, a.positions,
                         a.first_pos, a.last_pos, a.T, a.W, a.width};
    const int n = vec ? 4 : 1, cols = (a.width + n - 1) / n;
    const dim3 g((cols + 255) / 256, (a.T + kBlendRun - 1) / kBlendRun);
#define STK_BLEND(N, B) launch_pdl(shift_blend_kernel<A, N, B>, g, dim3(256), 0, st, b)
    if (vec && a.blends == 5) STK_BLEND(4, 5);
    else if (vec) STK_BLEND(4, 0);
    else if (a.blends == 5) STK_BLEND(1, 5);
    else STK_BLEND(1, 0);
#undef STK_BLEND
    return cudaGetLastError() == cudaSuccess ? 0 : -4;
  }
  // runs: long enough that the two tokens formed again cost little, short enough to fill the SMs
  a.run = 1;
  if (!decode) {
    a.run = a.T / (2 * sm_count);
    a.run = a.run < 2 ? 2 : a.run > 16 ? 16 : a.run;
  }
  const int need = (a.W + (vec ? 4 : 1) - 1) / (vec ? 4 : 1);
  const int threads = need <= 256 ? 256 : need <= 512 ? 512 : 1024, its = (need + threads - 1) / threads;
  const dim3 grid((a.T + a.run - 1) / a.run);
#define STK_SHIFT(N, NIT)                                                                                             \
  do {                                                                                                                \
    if (threads == 256) launch_pdl(shifted_norm_kernel<A, N, NIT, 256>, grid, dim3(threads), 0, st, a);               \
    else launch_pdl(shifted_norm_kernel<A, N, NIT, 1024>, grid, dim3(threads), 0, st, a);                             \
  } while (0)
  if (vec) {
    if (its == 1) STK_SHIFT(4, 1);
    else if (its <= 4) STK_SHIFT(4, 4);
    else return -2;
  } else {
    if (its == 1) STK_SHIFT(1, 1);
    else if (its <= 16) STK_SHIFT(1, 16);
    else return -2;
  }
#undef STK_SHIFT
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

__global__ void __launch_bounds__(256)
shift_commit_kernel(const int* __restrict__ query_start, const int* __restrict__ req_rows, const int64_t* __restrict__ ids,
                    int64_t* __restrict__ token, const float* __restrict__ then, float* __restrict__ now, int n_rows, long long n) {
  pdl_wait();
  pdl_trigger();
  const int ri = blockIdx.x, layer = blockIdx.y;
  const int end = query_start[ri + 1];
  if (end <= query_start[ri]) return;
  const int row = req_rows[ri];
  if (row < 0) return;
  if (layer == 0 && threadIdx.x == 0) token[row] = ids[end - 1];
  const long long at = (static_cast<long long>(layer) * n_rows + row) * n;
  if ((n & 3) == 0) {
    for (long long i = threadIdx.x * 4; i < n; i += blockDim.x * 4)
      *reinterpret_cast<float4*>(now + at + i) = *reinterpret_cast<const float4*>(then + at + i);
  } else {
    for (long long i = threadIdx.x; i < n; i += blockDim.x) now[at + i] = then[at + i];
  }
}

}  // namespace stk

using namespace stk;

// table null: no bigram embedding.
STK_API int stk_embed_bigram(const int64_t* ids, const void* embed, int embed_fp32, float scale, const void* table, int buckets, int mul_prev,
                             int mul_cur, const int* tok_req, const int64_t* positions, const int* first_pos, const int64_t* last_token,
                             float* x, int T, int W, int vocab, int* status, void* stream) {
  if (T <= 0) return 0;
  if (buckets < 1 || mul_prev < 0 || mul_cur < 0) return -1;
  cudaStream_t st = (cudaStream_t)stream;
  if (embed_fp32)
    launch_pdl(embed_bigram_kernel<float>, dim3(T), dim3(256), 0, st, ids, (const float*)embed, scale, (const float*)table, buckets, mul_prev,
               mul_cur, tok_req, positions, first_pos, last_token, x, W, vocab, status);
  else
    launch_pdl(embed_bigram_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, st, ids, (const __nv_bfloat16*)embed, scale,
               (const __nv_bfloat16*)table, buckets, mul_prev, mul_cur, tok_req, positions, first_pos, last_token, x, W, vocab, status);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// y0, y1: mixer outputs (w: weight of their RMS norm, null for none); ff [T, W] fp32 rows or pairs: a token's `top` expert rows; all may be
// null.  x_out null: the sum is not kept.  inv: work space [T] (or null).  shift null: h only; rows: of these T rows.  decode: every span is one token.
STK_API int stk_shifted_norm(const float* x, float* x_out, const float* y0, long long ld0, const float* w0, float f0, const float* y1,
                             long long ld1, const float* w1, float f1, const float* ff, long long ldf, const void* pairs, long long ldp,
                             const int* pair_row, const float* weights, int top, const float* norm, float eps, const float* shift,
                             const float* mu, int blends, void* h, void* s, void* mix, int width, int fp32, const float* now, float* then,
                             const int* tok_req, const int64_t* positions, const int* first_pos, const int* last_pos, const int64_t* rows,
                             float* inv, int T, int W, int decode, int sm_count, void* stream) {
  if (T <= 0) return 0;
  if (top > 32 || (pairs != nullptr && ff != nullptr) || (shift != nullptr && rows != nullptr) || blends < 0 || (rows != nullptr && x_out != nullptr) ||
      x == x_out)
    return -1;
  const ShiftOut o0{y0, ld0, w0, f0}, o1{y1, ld1, w1, f1};
  if (fp32) {
    const ShiftArgs<float> a{x, x_out, {o0, o1}, ff, ldf, (const float*)pairs, ldp, pair_row, weights, top, norm, eps, shift, mu, blends,
                             (float*)h, (float*)s, (float*)mix, now, then, tok_req, positions, first_pos, last_pos, rows, T, W, width, 1, nullptr};
    return launch_shifted(a, inv, decode, sm_count, (cudaStream_t)stream);
  }
  const ShiftArgs<__nv_bfloat16> a{x, x_out, {o0, o1}, ff, ldf, (const __nv_bfloat16*)pairs, ldp, pair_row, weights, top, norm, eps, shift, mu,
                                   blends, (__nv_bfloat16*)h, (__nv_bfloat16*)s, (__nv_bfloat16*)mix, now, then, tok_req, positions,
                                   first_pos, last_pos, rows, T, W, width, 1, nullptr};
  return launch_shifted(a, inv, decode, sm_count, (cudaStream_t)stream);
}

// then, now [layers, n_rows, n].
STK_API int stk_shift_commit(const int* query_start, const int* req_rows, int n_req, const int64_t* ids, int64_t* token, const float* then,
                             float* now, int layers, int n_rows, int n, void* stream) {
  if (n_req <= 0) return 0;
  if (layers < 1 || layers > 65535) return -1;
  launch_pdl(shift_commit_kernel, dim3(n_req, layers), dim3(256), 0, (cudaStream_t)stream, query_start, req_rows, ids, token, then, now, n_rows,
             static_cast<long long>(n));
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
