// Latent attention over the paged latent cache.
//
// A cached row holds one token's latent c (rank values) and the rotated key part shared by all heads. Two forms of the same
// attention:
//  * absorbed: queries are taken into latent space (W_uk^T q), scores and outputs are products with the cached rows
//    themselves, all heads of a token reading the same bytes; W_uv brings the result back. Decoding uses it: the cache is
//    the only thing that grows with the context, and it is read once for all heads.
//  * materialised (cached_prefill.cu): keys and values of the visible range are projected once, which needs far fewer
//    operations when many queries share them. Prompts use it.
// This file has the query / output projections around the absorbed form (whose kernels are those of cached_attention.cu) and the
// query layout of the materialised one.
#include <float.h>

#include "hybrid.h"
#include "hybrid_mma.cuh"

namespace mb {
namespace {

using namespace hy;

constexpr int TT = 8;  // rows that share the weight reads of a projection block

// ------------------------------------------------------------------------------------------------ projections
// Rotated part and padding of row t, head h (all threads of the block, rows t0 .. t0 + TT).
template <typename T, typename O>
__device__ __forceinline__ void absorb_rotated(const HyLatent& a, const T* __restrict__ q, const int* __restrict__ positions, int n_rows,
                                               O* __restrict__ ql, int qld, int h, int t0) {
  const int tail = qld - a.rank;
  for (int i = threadIdx.x; i < TT * tail; i += blockDim.x) {
    const int b = i / tail, c = i - b * tail, t = t0 + b;
    if (t >= n_rows) break;
    float v = 0.f;
    if (c < a.rot) {
      const T* src = q + (static_cast<long long>(t) * a.heads + h) * (a.dim + a.rot) + a.dim;
      float sn, cs;
      sincosf(static_cast<float>(positions[t]) * a.freq[c >> 1], &sn, &cs);
      const float u = to_f(src[c & ~1]), w = to_f(src[c | 1]);
      v = (c & 1) ? w * cs + u * sn : u * cs - w * sn;
    }
    ql[(static_cast<long long>(t) * a.heads + h) * qld + a.rank + c] = from_f<O>(v);
  }
}

// Block (x, head, row tile): x < nr: 128 latent columns; x == nr: the rotated part and the padding. VEC: 16 lanes cover the
// columns (16 bytes each), the block's 16 half-warps split the head's dimensions so that all weight loads are in flight at
// once; the partial sums meet in shared memory.
template <typename T, typename O, bool VEC>
__global__ void __launch_bounds__(256) absorb_q_kernel(const HyLatent a, const T* __restrict__ q, const int* __restrict__ positions,
                                                       int n_rows, O* __restrict__ ql, int qld, int nr) {
  extern __shared__ float qs[];  // [TT][dim], VEC: then [8][TT][128] partial sums
  const int h = blockIdx.y, t0 = blockIdx.z * TT, qd = a.dim + a.rot;
  if (static_cast<int>(blockIdx.x) == nr) {
    absorb_rotated<T, O>(a, q, positions, n_rows, ql, qld, h, t0);
    return;
  }
  for (int i = threadIdx.x; i < TT * a.dim; i += blockDim.x) {
    const int b = i / a.dim, d = i - b * a.dim;
    qs[i] = t0 + b < n_rows ? to_f(q[(static_cast<long long>(t0 + b) * a.heads + h) * qd + d]) : 0.f;
  }
  const T* w = static_cast<const T*>(a.ukv) + static_cast<long long>(h) * a.dim * a.rank;
  if constexpr (VEC) {
    float* part = qs + TT * a.dim;
    const int lane16 = threadIdx.x & 15, slice = threadIdx.x >> 4;  // 16 slices of the dimensions
    const int r = blockIdx.x * 128 + lane16 * 8;
    float acc[TT][8];
#pragma unroll
    for (int b = 0; b < TT; ++b)
#pragma unroll
      for (int k = 0; k < 8; ++k) acc[b][k] = 0.f;
    constexpr int U = 4;
    __syncthreads();
    if (r < a.rank) {
      for (int d0 = slice; d0 < a.dim; d0 += 16 * U) {
        uint4 raw[U];
#pragma unroll
        for (int u = 0; u < U; ++u)
          if (d0 + 16 * u < a.dim) raw[u] = *reinterpret_cast<const uint4*>(w + static_cast<long long>(d0 + 16 * u) * a.rank + r);
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int d = d0 + 16 * u;
          if (d >= a.dim) break;
          const uint32_t x4[4] = {raw[u].x, raw[u].y, raw[u].z, raw[u].w};
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x4[k]));
#pragma unroll
            for (int b = 0; b < TT; ++b) {
              const float qv = qs[b * a.dim + d];
              acc[b][2 * k] += f.x * qv;
              acc[b][2 * k + 1] += f.y * qv;
            }
          }
        }
      }
    }
    const int warp = threadIdx.x >> 5;
#pragma unroll
    for (int b = 0; b < TT; ++b)
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const float v = acc[b][k] + __shfl_xor_sync(0xffffffffu, acc[b][k], 16);
        if ((threadIdx.x & 16) == 0) part[(warp * TT + b) * 128 + lane16 * 8 + k] = v;
      }
    __syncthreads();
    for (int i = threadIdx.x; i < TT * 128; i += blockDim.x) {
      const int b = i >> 7, c = i & 127, rr = blockIdx.x * 128 + c;
      if (t0 + b >= n_rows || rr >= a.rank) continue;
      float v = 0.f;
#pragma unroll
      for (int k = 0; k < 8; ++k) v += part[(k * TT + b) * 128 + c];
      ql[(static_cast<long long>(t0 + b) * a.heads + h) * qld + rr] = from_f<O>(v);
    }
  } else {
    __syncthreads();
    const int r = blockIdx.x * 128 + threadIdx.x;
    if (threadIdx.x >= 128 || r >= a.rank) return;
    float acc[TT];
#pragma unroll
    for (int b = 0; b < TT; ++b) acc[b] = 0.f;
#pragma unroll 8
    for (int d = 0; d < a.dim; ++d) {
      const float v = to_f(w[static_cast<long long>(d) * a.rank + r]);
#pragma unroll
      for (int b = 0; b < TT; ++b) acc[b] += v * qs[b * a.dim + d];
    }
#pragma unroll
    for (int b = 0; b < TT; ++b)
      if (t0 + b < n_rows) ql[(static_cast<long long>(t0 + b) * a.heads + h) * qld + r] = from_f<O>(acc[b]);
  }
}

// Block (x, head, row tile): 32 output values of a head. o is [T, heads, splits, rank] with (max, sum) per split when ml is
// given (unnormalised partial outputs), else normalised and splits = 1. RT rows per block.
template <typename T, int RT>
__global__ void __launch_bounds__(256) latent_up_kernel(const HyLatent a, const float* __restrict__ o, const float* __restrict__ ml,
                                                        int splits, int n_rows, T* __restrict__ cat, int ldc, bool vec) {
  extern __shared__ float os[];  // [RT][rank]
  __shared__ float coef[RT][64];
  const int h = blockIdx.y, t0 = blockIdx.z * RT;
  const int rows = min(RT, n_rows - t0);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* wv = static_cast<const T*>(a.ukv) + (static_cast<long long>(a.heads) * a.dim + h * a.vdim) * a.rank;
  constexpr int N = Vec<T>::N, VB = 4, WC = 2;  // a warp's four output values; chunks of their weights fetched ahead
  const int v0 = blockIdx.x * 32 + warp * VB;
  float w[VB][WC][N];
  auto fetch = [&](int base) {
#pragma unroll
    for (int i = 0; i < VB; ++i)
#pragma unroll
      for (int k = 0; k < WC; ++k) {
        const int r = base + (k * 32 + lane) * N;
        if (v0 + i < a.vdim && r < a.rank) {
          Vec<T>::load(wv + static_cast<long long>(v0 + i) * a.rank + r, w[i][k]);
        } else {
#pragma unroll
          for (int j = 0; j < N; ++j) w[i][k][j] = 0.f;
        }
      }
  };
  if (vec) fetch(0);  // (does not depend on the attention's result)
  if (ml) {  // a warp per row: coefficients of the splits
    for (int b = warp; b < rows; b += 8) {
      const float* p = ml + (static_cast<long long>(t0 + b) * a.heads + h) * splits * 2;
      float mv[2], lv[2], m = -FLT_MAX;
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int s = lane + 32 * k;
        mv[k] = s < splits ? p[2 * s] : -FLT_MAX;
        lv[k] = s < splits ? p[2 * s + 1] : 0.f;
        m = fmaxf(m, mv[k]);
      }
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, off));
      float l = 0.f, c[2];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        c[k] = mv[k] == -FLT_MAX ? 0.f : exp2f(mv[k] - m);
        l += c[k] * lv[k];
      }
      l = warp_sum(l);
      const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
      for (int k = 0; k < 2; ++k)
        if (lane + 32 * k < splits) coef[b][lane + 32 * k] = c[k] * inv;
    }
    __syncthreads();
  }
  if ((a.rank & 3) == 0) {
    for (int i = threadIdx.x * 4; i < RT * a.rank; i += blockDim.x * 4) {
      const int b = i / a.rank, r = i - b * a.rank;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (b < rows) {
        const float* p = o + (static_cast<long long>(t0 + b) * a.heads + h) * splits * a.rank + r;
        if (ml) {
#pragma unroll 4
          for (int s = 0; s < splits; ++s) {
            const float c = coef[b][s];
            const float4 u = *reinterpret_cast<const float4*>(p + static_cast<long long>(s) * a.rank);
            v.x += c * u.x; v.y += c * u.y; v.z += c * u.z; v.w += c * u.w;
          }
        } else {
          v = *reinterpret_cast<const float4*>(p);
        }
      }
      *reinterpret_cast<float4*>(os + i) = v;
    }
  } else {
    for (int i = threadIdx.x; i < RT * a.rank; i += blockDim.x) {
      const int b = i / a.rank, r = i - b * a.rank;
      float v = 0.f;
      if (b < rows) {
        const float* p = o + (static_cast<long long>(t0 + b) * a.heads + h) * splits * a.rank + r;
        if (ml) {
          for (int s = 0; s < splits; ++s) v += coef[b][s] * p[static_cast<long long>(s) * a.rank];
        } else {
          v = p[0];
        }
      }
      os[i] = v;
    }
  }
  __syncthreads();
  float acc[VB][RT];
#pragma unroll
  for (int i = 0; i < VB; ++i)
#pragma unroll
    for (int b = 0; b < RT; ++b) acc[i][b] = 0.f;
  if (vec) {
    for (int base = 0; base < a.rank; base += WC * 32 * N) {
      if (base > 0) fetch(base);
#pragma unroll
      for (int k = 0; k < WC; ++k) {
        const int r = base + (k * 32 + lane) * N;
        if (r >= a.rank) continue;
#pragma unroll
        for (int b = 0; b < RT; ++b) {
          float x[N];
#pragma unroll
          for (int j = 0; j < N; j += 4) {
            const float4 u = *reinterpret_cast<const float4*>(os + b * a.rank + r + j);
            x[j] = u.x; x[j + 1] = u.y; x[j + 2] = u.z; x[j + 3] = u.w;
          }
#pragma unroll
          for (int i = 0; i < VB; ++i)
#pragma unroll
            for (int j = 0; j < N; ++j) acc[i][b] += w[i][k][j] * x[j];
        }
      }
    }
  } else {
    for (int r = lane; r < a.rank; r += 32)
#pragma unroll
      for (int i = 0; i < VB; ++i) {
        const float x = v0 + i < a.vdim ? to_f(wv[static_cast<long long>(v0 + i) * a.rank + r]) : 0.f;
#pragma unroll
        for (int b = 0; b < RT; ++b) acc[i][b] += x * os[b * a.rank + r];
      }
  }
#pragma unroll
  for (int i = 0; i < VB; ++i)
#pragma unroll
    for (int b = 0; b < RT; ++b) {
      const float v = warp_sum(acc[i][b]);
      if (lane == 0 && b < rows && v0 + i < a.vdim) cat[static_cast<long long>(t0 + b) * ldc + h * a.vdim + v0 + i] = from_f<T>(v);
    }
}

// ------------------------------------------------------------------------------------------------ projections of many rows
// Tensor-core forms of the two per-head projections (bf16, more rows than the kernels above share a weight read among).
constexpr int HM = 32;    // rows per CTA
constexpr int AN = 128;   // latent columns per CTA (queries into latent space)
constexpr int UN = 32;    // output values per CTA (latent outputs back)

// ql[t, h, r] = sum_d q[t, h, d] W_uk[h * dim + d, r]; the block after the last column tile writes rotated part and padding.
template <typename O>
__global__ void __launch_bounds__(128) absorb_mma_kernel(const HyLatent a, const bf16* __restrict__ q, const int* __restrict__ positions,
                                                         int n_rows, O* __restrict__ ql, int qld, int nr) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int h = blockIdx.y, t0 = blockIdx.z * HM, qd = a.dim + a.rot;
  if (static_cast<int>(blockIdx.x) == nr) {
    for (int t = t0; t < min(n_rows, t0 + HM); t += TT) absorb_rotated<bf16, O>(a, q, positions, min(n_rows, t0 + HM), ql, qld, h, t);
    return;
  }
  const int DP = (a.dim + 15) / 16 * 16, lda = DP + 8, ldb = AN + 8, r0 = blockIdx.x * AN;
  bf16* As = reinterpret_cast<bf16*>(raw);  // [HM][lda]
  bf16* Bs = As + HM * lda;                 // [DP][ldb]
  for (int i = threadIdx.x; i < HM * (DP / 8); i += 128) {
    const int r = i / (DP / 8), c = (i - r * (DP / 8)) * 8;
    const bool ok = t0 + r < n_rows && c < a.dim;
    cp16(s_u32(As + r * lda + c), q + (ok ? (static_cast<long long>(t0 + r) * a.heads + h) * qd + c : 0), ok ? 16 : 0);
  }
  const bf16* w = static_cast<const bf16*>(a.ukv) + static_cast<long long>(h) * a.dim * a.rank;
  for (int i = threadIdx.x; i < DP * (AN / 8); i += 128) {
    const int d = i / (AN / 8), c = (i & (AN / 8 - 1)) * 8;
    const bool ok = d < a.dim && r0 + c < a.rank;
    cp16(s_u32(Bs + d * ldb + c), w + (ok ? static_cast<long long>(d) * a.rank + r0 + c : 0), ok ? 16 : 0);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wm = warp & 1, wn = warp >> 1;
  float acc[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll 2
  for (int k0 = 0; k0 < DP; k0 += 16) {
    uint32_t af[4];
    ldsm4(s_u32(As + (wm * 16 + (lane & 15)) * lda + k0 + ((lane >> 4) << 3)), af);
#pragma unroll
    for (int jp = 0; jp < 4; ++jp) {
      uint32_t b[4];
      ldsm4t(s_u32(Bs + (k0 + (lane & 7) + (((lane >> 3) & 1) << 3)) * ldb + wn * 64 + jp * 16 + ((lane >> 4) << 3)), b);
      mma(acc[2 * jp], af, b[0], b[1]);
      mma(acc[2 * jp + 1], af, b[2], b[3]);
    }
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int r = r0 + wn * 64 + j * 8 + (lane & 3) * 2;
    if (r >= a.rank) continue;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = t0 + wm * 16 + (lane >> 2) + e * 8;
      if (t >= n_rows) continue;
      O* dst = ql + (static_cast<long long>(t) * a.heads + h) * qld + r;
      dst[0] = from_f<O>(acc[j][2 * e]);
      dst[1] = from_f<O>(acc[j][2 * e + 1]);
    }
  }
}

// cat[t, h * vdim + v] = sum_r o[t, h, r] W_uv[h * vdim + v, r] over the merged split outputs (ml) or normalised ones.
__global__ void __launch_bounds__(128) up_mma_kernel(const HyLatent a, const float* __restrict__ o, const float* __restrict__ ml,
                                                     int splits, int n_rows, bf16* __restrict__ cat, int ldc) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float coef[HM][64];
  const int h = blockIdx.y, t0 = blockIdx.z * HM, v0 = blockIdx.x * UN, rows = min(HM, n_rows - t0);
  const int KP = (a.rank + 15) / 16 * 16, ld = KP + 8;
  bf16* As = reinterpret_cast<bf16*>(raw);  // [HM][ld]
  bf16* Bs = As + HM * ld;                  // [UN][ld]
  const bf16* w = static_cast<const bf16*>(a.ukv) + (static_cast<long long>(a.heads) * a.dim + h * a.vdim) * a.rank;
  for (int i = threadIdx.x; i < UN * (KP / 8); i += 128) {
    const int v = i / (KP / 8), c = (i - v * (KP / 8)) * 8;
    const bool ok = v0 + v < a.vdim && c < a.rank;
    cp16(s_u32(Bs + v * ld + c), w + (ok ? static_cast<long long>(v0 + v) * a.rank + c : 0), ok ? 16 : 0);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (static_cast<int>(threadIdx.x) < HM) {
    const int b = threadIdx.x;
    if (b < rows) {
      float l = 0.f, m = -FLT_MAX;
      if (ml) {
        const float* p = ml + (static_cast<long long>(t0 + b) * a.heads + h) * splits * 2;
        for (int s = 0; s < splits; ++s) m = fmaxf(m, p[2 * s]);
        for (int s = 0; s < splits; ++s) {
          const float c = p[2 * s] == -FLT_MAX ? 0.f : exp2f(p[2 * s] - m);
          coef[b][s] = c;
          l += c * p[2 * s + 1];
        }
        l = l > 0.f ? 1.f / l : 0.f;
        for (int s = 0; s < splits; ++s) coef[b][s] *= l;
      } else {
        coef[b][0] = 1.f;
      }
    }
  }
  __syncthreads();
  for (int i = threadIdx.x * 4; i < HM * KP; i += 128 * 4) {
    const int b = i / KP, r = i - b * KP;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (b < rows && r < a.rank) {
      const float* p = o + (static_cast<long long>(t0 + b) * a.heads + h) * splits * a.rank + r;
#pragma unroll 2
      for (int s = 0; s < splits; ++s) {
        const float c = coef[b][s];
        const float4 u = *reinterpret_cast<const float4*>(p + static_cast<long long>(s) * a.rank);
        v.x += c * u.x; v.y += c * u.y; v.z += c * u.z; v.w += c * u.w;
      }
    }
    const __nv_bfloat162 x = __floats2bfloat162_rn(v.x, v.y), y = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(As + b * ld + r) = make_uint2(*reinterpret_cast<const uint32_t*>(&x), *reinterpret_cast<const uint32_t*>(&y));
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  const int wm = warp & 1, wn = warp >> 1;
  float acc[2][4];
#pragma unroll
  for (int j = 0; j < 2; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll 4
  for (int k0 = 0; k0 < KP; k0 += 16) {
    uint32_t af[4], b[4];
    ldsm4(s_u32(As + (wm * 16 + (lane & 15)) * ld + k0 + ((lane >> 4) << 3)), af);
    ldsm4(s_u32(Bs + (wn * 16 + (lane & 7) + ((lane >> 4) << 3)) * ld + k0 + (((lane >> 3) & 1) << 3)), b);
    mma(acc[0], af, b[0], b[1]);
    mma(acc[1], af, b[2], b[3]);
  }
#pragma unroll
  for (int j = 0; j < 2; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int v = v0 + wn * 16 + j * 8 + (lane & 3) * 2 + (e & 1), t = wm * 16 + (lane >> 2) + (e >> 1) * 8;
      if (v < a.vdim && t < rows) cat[static_cast<long long>(t0 + t) * ldc + h * a.vdim + v] = __float2bfloat16(acc[j][e]);
    }
}

// ------------------------------------------------------------------------------------------------ materialised form: inputs
__global__ void __launch_bounds__(256) pad_q_kernel(const HyLatent a, const bf16* __restrict__ q, const int* __restrict__ positions,
                                                    bf16* __restrict__ out, int nope, int rot) {
  const long long t = blockIdx.x;
  const int per = (nope + rot) / 8, qd = a.dim + a.rot;
  const float pos = static_cast<float>(positions[t]);
  for (int i = threadIdx.x; i < a.heads * per; i += blockDim.x) {
    const int h = i / per, c = (i - h * per) * 8;
    const bf16* src = q + (t * a.heads + h) * qd;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (c < nope) {
      if (c < a.dim) v = *reinterpret_cast<const uint4*>(src + c);
    } else if (c - nope < a.rot) {
      float x[8];
      Vec<bf16>::load(src + a.dim + c - nope, x);
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        float sn, cs;
        sincosf(pos * a.freq[(c - nope) / 2 + k], &sn, &cs);
        const float u = x[2 * k], w = x[2 * k + 1];
        x[2 * k] = u * cs - w * sn;
        x[2 * k + 1] = w * cs + u * sn;
      }
      Vec<bf16>::store(out + (t * a.heads + h) * (nope + rot) + c, x);
      continue;
    }
    *reinterpret_cast<uint4*>(out + (t * a.heads + h) * (nope + rot) + c) = v;
  }
}

template <typename T, typename O>
int absorb_t(const HyLatent& a, const void* q, const int* positions, int n, void* ql, int qld, cudaStream_t s) {
  const int nr = (a.rank + 127) / 128;
  auto go = [&](auto kern, size_t smem) -> int {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    kern<<<dim3(nr + 1, a.heads, (n + TT - 1) / TT), 256, smem, s>>>(a, static_cast<const T*>(q), positions, n, static_cast<O*>(ql), qld, nr);
    return static_cast<int>(cudaGetLastError());
  };
  if constexpr (sizeof(T) == 2) {
    const int DP = (a.dim + 15) / 16 * 16;
    const size_t sm = sizeof(bf16) * (HM * (DP + 8) + DP * (AN + 8));
    if (n > TT && a.rank % 8 == 0 && a.dim % 8 == 0 && a.rot % 8 == 0 && sm <= 200 * 1024 && aligned16<T>(a.ukv, a.rank) && aligned16<T>(q, 8)) {
      auto kern = absorb_mma_kernel<O>;
      cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(sm));
      if (e != cudaSuccess) return static_cast<int>(e);
      kern<<<dim3(nr + 1, a.heads, (n + HM - 1) / HM), 128, sm, s>>>(a, static_cast<const T*>(q), positions, n, static_cast<O*>(ql), qld, nr);
      return static_cast<int>(cudaGetLastError());
    }
    if (a.rank % 8 == 0 && aligned16<T>(a.ukv, a.rank)) return go(absorb_q_kernel<T, O, true>, sizeof(float) * (TT * a.dim + 8 * TT * 128));
  }
  return go(absorb_q_kernel<T, O, false>, sizeof(float) * TT * a.dim);
}

template <typename T, int RT>
int up_rt(const HyLatent& a, const float* o, const float* ml, int splits, int n, void* cat, int ldc, cudaStream_t s) {
  const size_t smem = sizeof(float) * RT * a.rank;
  auto kern = latent_up_kernel<T, RT>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3((a.vdim + 31) / 32, a.heads, (n + RT - 1) / RT), 256, smem, s>>>(a, o, ml, splits, n, static_cast<T*>(cat), ldc,
                                                                              a.rank % Vec<T>::N == 0 && aligned16<T>(a.ukv, a.rank));
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int up_t(const HyLatent& a, const float* o, const float* ml, int splits, int n, void* cat, int ldc, cudaStream_t s) {
  if constexpr (sizeof(T) == 2) {
    const size_t sm = sizeof(bf16) * (HM + UN) * static_cast<size_t>((a.rank + 15) / 16 * 16 + 8);
    if (n > TT && a.rank % 8 == 0 && sm <= 200 * 1024 && aligned16<T>(a.ukv, a.rank)) {
      cudaError_t e = cudaFuncSetAttribute(up_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(sm));
      if (e != cudaSuccess) return static_cast<int>(e);
      up_mma_kernel<<<dim3((a.vdim + UN - 1) / UN, a.heads, (n + HM - 1) / HM), 128, sm, s>>>(a, o, ml, splits, n, static_cast<T*>(cat), ldc);
      return static_cast<int>(cudaGetLastError());
    }
  }
  return n <= 2 ? up_rt<T, 1>(a, o, ml, splits, n, cat, ldc, s) : up_rt<T, 4>(a, o, ml, splits, n, cat, ldc, s);
}

}  // namespace

int hy_absorb_q(bool f32, const HyLatent& a, const void* q, const int* positions, int T, void* ql, int qld, bool out_f32,
                cudaStream_t s) {
  if (f32) return absorb_t<float, float>(a, q, positions, T, ql, qld, s);
  if (out_f32) return absorb_t<bf16, float>(a, q, positions, T, ql, qld, s);
  return absorb_t<bf16, bf16>(a, q, positions, T, ql, qld, s);
}

HyAttend hy_latent_view(const HyLatent& a) {
  HyAttend v = {};
  static_cast<HyCache&>(v) = a;
  v.heads = v.group = a.heads;   // all heads read the same row: scores over all of it, outputs of its first `rank` columns
  v.kd = a.rank + a.rot;
  v.vd = a.rank;
  v.window = a.window;
  v.scale = a.scale;
  return v;
}

int hy_latent_up(bool f32, const HyLatent& a, const float* o, const float* ml, int splits, int T, void* cat, int ldc, cudaStream_t s) {
  if (splits < 1 || splits > 64) return static_cast<int>(cudaErrorInvalidValue);
  return f32 ? up_t<float>(a, o, ml, splits, T, cat, ldc, s) : up_t<bf16>(a, o, ml, splits, T, cat, ldc, s);
}

int hy_pad_q(const HyLatent& a, const void* q, const int* positions, int T, int nope_pad, int rot_pad, void* out, cudaStream_t s) {
  pad_q_kernel<<<T, 256, 0, s>>>(a, static_cast<const bf16*>(q), positions, static_cast<bf16*>(out), nope_pad, rot_pad);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace mb
