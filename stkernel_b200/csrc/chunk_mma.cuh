// Building blocks of the chunked recurrences (mlstm.cu, linear_scan.cu): warp-level bf16 products, fp32 operands as bf16 pairs, chunk
// numbering over the spans of a step, token tiles into shared memory.
#pragma once
#include "common.cuh"

namespace stk {

constexpr int kChunk = 64;
constexpr int kStStride = 72;                    // shared-memory row stride of a 64-column tile

__device__ __forceinline__ void mls_ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mls_ldsm4_t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mls_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mls_split(float x, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16(x);
  lo = __float2bfloat16(x - bf16_to_f(hi));
}
__device__ __forceinline__ void mls_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 r = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&r);
}

// chunk index of the step -> (request, first chunk of the request, tokens [t0, t0 + n) of the step); false past the end
struct ChunkRef { int ri, first, t0, n; };
__device__ __forceinline__ bool find_chunk(const int* query_start, int n_req, int min_span, int ci, ChunkRef& c) {
  int base = 0;
  for (int i = 0; i < n_req; ++i) {
    const int q0 = query_start[i], span = query_start[i + 1] - q0;
    if (span < min_span) continue;
    const int nc = (span + kChunk - 1) / kChunk;
    if (ci < base + nc) {
      c.ri = i;
      c.first = base;
      c.t0 = q0 + (ci - base) * kChunk;
      c.n = min(kChunk, span - (ci - base) * kChunk);
      return true;
    }
    base += nc;
  }
  return false;
}

// rows [0, 64) x cols [0, width) of head columns into shared memory; rows >= n and columns >= width up to `cols` are zero
__device__ __forceinline__ void load_rows(__nv_bfloat16* dst, int stride, int cols, const __nv_bfloat16* src, long long ld, int n,
                                          int width, int nthreads) {
  if ((width & 7) == 0 && (cols & 7) == 0 && (ld & 7) == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0) {
    const int ch = cols >> 3;
    for (int e = threadIdx.x; e < kChunk * ch; e += nthreads) {
      const int r = e / ch, c = (e - r * ch) * 8;
      uint4 v = make_uint4(0, 0, 0, 0);
      if (r < n && c < width) v = *reinterpret_cast<const uint4*>(src + r * ld + c);
      *reinterpret_cast<uint4*>(dst + r * stride + c) = v;
    }
  } else {
    for (int e = threadIdx.x; e < kChunk * cols; e += nthreads) {
      const int r = e / cols, c = e - r * cols;
      dst[r * stride + c] = r < n && c < width ? src[r * ld + c] : __float2bfloat16(0.f);
    }
  }
}

__device__ __forceinline__ void mls_cp16(void* dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void mls_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void mls_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Like load_rows, but asynchronous when the rows are 16-byte aligned.
__device__ __forceinline__ void load_rows_async(__nv_bfloat16* dst, int stride, int cols, const __nv_bfloat16* src, long long ld,
                                                int n, int width, int nthreads) {
  if ((width & 7) == 0 && (cols & 7) == 0 && (ld & 7) == 0 && (reinterpret_cast<uintptr_t>(src) & 15) == 0) {
    const int ch = cols >> 3;
    for (int e = threadIdx.x; e < kChunk * ch; e += nthreads) {
      const int r = e / ch, c = (e - r * ch) * 8;
      const bool ok = r < n && c < width;
      mls_cp16(dst + r * stride + c, ok ? src + r * ld + c : src, ok);
    }
  } else {
    load_rows(dst, stride, cols, src, ld, n, width, nthreads);
  }
}

// chunks of request ri begin at this index of the step's chunk numbering
__device__ __forceinline__ int first_chunk(const int* query_start, int min_span, int ri) {
  int first = 0;
  for (int i = 0; i < ri; ++i) {
    const int s = query_start[i + 1] - query_start[i];
    if (s >= min_span) first += (s + kChunk - 1) / kChunk;
  }
  return first;
}

}  // namespace stk
