// Tensor-core fragments (mma.sync), asynchronous tile copies and two-term bf16 splits of the planned-layer kernels.
#pragma once
#include "hybrid_common.cuh"

namespace mb {
namespace hy {

__device__ __forceinline__ uint32_t s_u32(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// fp32 pair -> two bf16 terms whose sum keeps 16 bits of mantissa
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_wait_all() {
  cp_commit();
  asm volatile("cp.async.wait_group 0;" ::: "memory");
}

constexpr float LOG2E = 1.4426950408889634f;

// rows [n, w] of a row-major bf16 matrix (pitch `pitch`) into smem [rows][ld], zero filled to wp columns; vec: by 16-byte
// asynchronous copies the caller waits for
template <int THREADS>
__device__ __forceinline__ void load_tile(const bf16* __restrict__ src, long long pitch, int n, int w, int rows, int wp, bf16* dst,
                                          int ld, bool vec) {
  if (vec) {
    const int per = wp / 8;
    if ((THREADS) % per == 0) {  // every thread keeps its column
      const int step = THREADS / per, r0 = threadIdx.x / per, c = (threadIdx.x - r0 * per) * 8;
      const bool col = c < w;
      const bf16* p = src + r0 * pitch + c;
      uint32_t d = s_u32(dst + r0 * ld + c);
#pragma unroll 4
      for (int r = r0; r < rows; r += step, p += step * pitch, d += step * ld * 2) {
        const bool ok = col && r < n;
        cp16(d, ok ? p : src, ok ? 16 : 0);
      }
      return;
    }
    for (int i = threadIdx.x; i < rows * per; i += THREADS) {
      const int r = i / per, c = (i - r * per) * 8;
      const bool ok = r < n && c < w;
      cp16(s_u32(dst + r * ld + c), src + (ok ? r * pitch + c : 0), ok ? 16 : 0);
    }
  } else {
    for (int i = threadIdx.x; i < rows * wp; i += THREADS) {
      const int r = i / wp, c = i - r * wp;
      dst[r * ld + c] = (r < n && c < w) ? src[r * pitch + c] : __float2bfloat16(0.f);
    }
  }
}

}  // namespace hy
}  // namespace mb
