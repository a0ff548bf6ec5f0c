// Latent attention over paged latent rows: the layer's small kernels and the form for any size and type.
//
//   latent_prep       norms of the query and the key/value latent, rotation of the shared key part, insertion of the row
//   latent_rows       cached rows of whole requests copied into one contiguous matrix (prompts expand keys and values from it)
//   latent_attn_simt  queries in latent space against the rows, fp32 arithmetic throughout: one CTA per (token, head)
//
// Queries are brought into latent space by the key expansion (q . W_uk c = W_uk^T q . c), so one row serves all heads as key
// and, up to the value expansion of the result, as value.
#define STK_PDL_CLASS 8
#include "latent_attention.cuh"

namespace stk {

struct PrepArgs {
  const float* p; long long ldp; int q_off, kv_off;      // fp32 projections; kv_off < 0: the layer caches nothing
  const float* wq; const float* wkv;                     // norm weights
  float eps;
  int Q, q_width, C, R;
  const int64_t* positions; const int* tok_req;
  const int* table; int bt_stride;
  void* cache; int row, rot_off;
  const float* freq;
  void* cq; long long ldcq;
};

// One CTA per token.  Threads of the first half norm the query latent, those of the second half the key/value latent.
template <typename A>
__global__ void __launch_bounds__(256)
latent_prep_kernel(const PrepArgs a) {
  __shared__ float part[8];
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const int half = threadIdx.x >> 7, i0 = threadIdx.x & 127;
  const int n = half ? (a.kv_off >= 0 ? a.C : 0) : a.Q;
  const float* src = a.p + t * a.ldp + (half ? (a.kv_off >= 0 ? a.kv_off : 0) : a.q_off);
  float v[16];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 16; ++j) {
    const int i = i0 + j * 128;
    v[j] = j * 128 < n && i < n ? src[i] : 0.f;
  }
#pragma unroll
  for (int j = 0; j < 16; ++j) {
    if (j * 128 >= n) break;
    ss = fmaf(v[j], v[j], ss);
  }
  for (int i = i0 + 16 * 128; i < n; i += 128) ss = fmaf(src[i], src[i], ss);
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = (part[half * 4] + part[half * 4 + 1]) + (part[half * 4 + 2] + part[half * 4 + 3]);
  if (half == 0) {
    const float inv = 1.f / sqrtf(ss / static_cast<float>(a.Q) + a.eps);
    A* o = reinterpret_cast<A*>(a.cq) + t * a.ldcq;
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      const int i = i0 + j * 128;
      if (j * 128 >= a.q_width) break;
      if (i < a.q_width) lat_st(o + i, i < a.Q ? v[j] * inv * a.wq[i] : 0.f);
    }
    for (int i = i0 + 16 * 128; i < a.q_width; i += 128) lat_st(o + i, i < a.Q ? src[i] * inv * a.wq[i] : 0.f);
    return;
  }
  if (a.kv_off < 0) return;
  const int req = a.tok_req[t];
  const long long pos = a.positions[t];
  if (req < 0 || pos < 0) return;
  const int page = a.table[static_cast<long long>(req) * a.bt_stride + pos / kLatPage];
  if (page < 0) return;
  const float inv = 1.f / sqrtf(ss / static_cast<float>(a.C) + a.eps);
  A* o = reinterpret_cast<A*>(a.cache) + (static_cast<long long>(page) * kLatPage + pos % kLatPage) * a.row;
#pragma unroll
  for (int j = 0; j < 16; ++j) {
    const int i = i0 + j * 128;
    if (j * 128 >= a.rot_off) break;
    if (i < a.rot_off) lat_st(o + i, i < a.C ? v[j] * inv * a.wkv[i] : 0.f);
  }
  for (int i = i0 + 16 * 128; i < a.rot_off; i += 128) lat_st(o + i, i < a.C ? src[i] * inv * a.wkv[i] : 0.f);
  const int pairs = a.R >> 1;
  for (int i = i0; i < pairs; i += 128) {
    const float2 w = cos_sin_split(pos, a.freq[i], a.freq[pairs + i]);
    const float x = src[a.C + 2 * i], y = src[a.C + 2 * i + 1];
    lat_st(o + a.rot_off + 2 * i, x * w.x - y * w.y);
    lat_st(o + a.rot_off + 2 * i + 1, y * w.x + x * w.y);
  }
  for (int i = a.rot_off + a.R + i0; i < a.row; i += 128) lat_st(o + i, 0.f);
}

// ---- any size, fp32 arithmetic ------------------------------------------------------------------
constexpr int kLatKeys = 512, kLatAcc = 16;

template <typename A>
__global__ void __launch_bounds__(128)
latent_attn_simt_kernel(const LatArgs a, const int* __restrict__ first_pos, const int* __restrict__ last_pos, int max_span) {
  __shared__ float q[2304];
  __shared__ float sc[kLatKeys];
  __shared__ float red[32];
  pdl_wait();
  pdl_trigger();
  const long long t = blockIdx.x;
  const int h = blockIdx.y;
  const int req = a.tok_req[t];
  const long long pos = a.positions[t];
  A* out = reinterpret_cast<A*>(a.out) + t * a.ldo + h * a.cp;
  if (req < 0 || pos < 0) {
    for (int d = threadIdx.x; d < a.cp; d += blockDim.x) lat_st(out + d, 0.f);
    return;
  }
  if (last_pos[t] - first_pos[t] + 1 > max_span) return;
  const A* qa = reinterpret_cast<const A*>(a.qa) + t * a.ldqa + h * a.cp;
  const A* qr = reinterpret_cast<const A*>(a.qr) + t * a.ldqr + h * a.R;
  for (int d = threadIdx.x; d < a.rot_off; d += blockDim.x) q[d] = d < a.C ? lat_f(qa[d]) : 0.f;
  const int pairs = a.R >> 1;
  for (int i = threadIdx.x; i < pairs; i += blockDim.x) {
    const float2 w = cos_sin_split(pos, a.freq[i], a.freq[pairs + i]);
    const float x = lat_f(qr[2 * i]), y = lat_f(qr[2 * i + 1]);
    q[a.rot_off + 2 * i] = x * w.x - y * w.y;
    q[a.rot_off + 2 * i + 1] = y * w.x + x * w.y;
  }
  for (int d = a.rot_off + a.R + threadIdx.x; d < a.row; d += blockDim.x) q[d] = 0.f;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int* bt = a.table + static_cast<long long>(req) * a.bt_stride;
  const A* cache = reinterpret_cast<const A*>(a.cache);
  auto row_of = [&](long long p) {
    const int page = bt[p / kLatPage];
    return cache + (static_cast<long long>(page < 0 ? 0 : page) * kLatPage + p % kLatPage) * a.row;
  };
  float m = -INFINITY, l = 0.f, acc[kLatAcc];
#pragma unroll
  for (int i = 0; i < kLatAcc; ++i) acc[i] = 0.f;
  for (long long k0 = 0; k0 <= pos; k0 += kLatKeys) {
    const int n = static_cast<int>(pos + 1 - k0 < kLatKeys ? pos + 1 - k0 : kLatKeys);
    float mx = -INFINITY;
    for (int j = warp; j < n; j += 4) {
      const A* r = row_of(k0 + j);
      float s = 0.f;
      for (int d = lane; d < a.row; d += 32) s = fmaf(q[d], lat_f(r[d]), s);
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
    for (int i = 0; i < kLatAcc; ++i) acc[i] *= f;
    for (int j = 0; j < n; ++j) {
      const A* r = row_of(k0 + j);
      const float p = sc[j];
#pragma unroll
      for (int i = 0; i < kLatAcc; ++i) {
        const int d = threadIdx.x + i * 128;
        if (d < a.C) acc[i] = fmaf(p, lat_f(r[d]), acc[i]);
      }
    }
    __syncthreads();
  }
  const float g = (a.gate != nullptr ? lat_sigmoid(a.gate[t * a.ldg + h]) : 1.f) / l;
#pragma unroll
  for (int i = 0; i < kLatAcc; ++i) {
    const int d = threadIdx.x + i * 128;
    if (d < a.cp) lat_st(out + d, d < a.C ? acc[i] * g : 0.f);
  }
}

}  // namespace stk

using namespace stk;

STK_API int stk_latent_prep(const float* p, long long ldp, int q_off, int kv_off, const float* wq, const float* wkv, float eps,
                            int q_rank, int q_width, int kv_rank, int rot, const int64_t* positions, const int* tok_req,
                            const int* table, int bt_stride, void* cache, int row, int rot_off, const float* freq, void* cq,
                            long long ldcq, int fp32, int T, void* stream) {
  if (T <= 0) return 0;
  if (q_rank < 1 || kv_rank < 1 || rot < 0 || (rot & 1) || rot_off < kv_rank || row < rot_off + rot || q_width < q_rank) return -1;
  PrepArgs a;
  a.p = p; a.ldp = ldp; a.q_off = q_off; a.kv_off = kv_off; a.wq = wq; a.wkv = wkv; a.eps = eps;
  a.Q = q_rank; a.q_width = q_width; a.C = kv_rank; a.R = rot; a.positions = positions; a.tok_req = tok_req;
  a.table = table; a.bt_stride = bt_stride; a.cache = cache; a.row = row; a.rot_off = rot_off; a.freq = freq;
  a.cq = cq; a.ldcq = ldcq;
  if (fp32) launch_pdl(latent_prep_kernel<float>, dim3(T), dim3(256), 0, (cudaStream_t)stream, a);
  else launch_pdl(latent_prep_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, (cudaStream_t)stream, a);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}

// Tokens whose span is at most max_span long.
STK_API int stk_latent_attention_simt(const void* qa, long long ldqa, int cp, const void* qr, long long ldqr, const float* gate,
                                      long long ldg, const int64_t* positions, const int* tok_req, const int* table,
                                      int bt_stride, const void* cache, int row, int rot_off, const float* freq, int heads,
                                      int kv_rank, int rot, float scale, void* out, long long ldo, int fp32,
                                      const int* first_pos, const int* last_pos, int max_span, int T, void* stream) {
  if (T <= 0) return 0;
  const LatArgs a = lat_args(qa, ldqa, cp, qr, ldqr, gate, ldg, positions, tok_req, table, bt_stride, cache, row, rot_off, freq,
                             heads, kv_rank, rot, scale, out, ldo);
  if (!lat_ok(a) || kv_rank > kLatAcc * 128 || cp > kLatAcc * 128 || heads > 65535) return -1;
  const dim3 grid(T, heads);
  if (fp32) launch_pdl(latent_attn_simt_kernel<float>, grid, dim3(128), 0, (cudaStream_t)stream, a, first_pos, last_pos, max_span);
  else launch_pdl(latent_attn_simt_kernel<__nv_bfloat16>, grid, dim3(128), 0, (cudaStream_t)stream, a, first_pos, last_pos, max_span);
  return cudaGetLastError() == cudaSuccess ? 0 : -4;
}
