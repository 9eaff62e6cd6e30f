// Mamba-2 mixer: causal convolution, selective state-space recurrence, single-token step.
//
//   S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,   dt = softplus(dt_raw + dt_bias)
//
// Three ways through the recurrence, all on the same per-sequence state [heads, P, N] in fp32:
//  * scan: token after token, a warp per state row (any sizes, fp32 throughout);
//  * chunks: 128 tokens at a time on the tensor cores. Within a chunk y = (C B^T o decay o dt) x, between chunks the state is
//    carried: (1) every chunk's own contribution to the state, (2) a scan over chunks, (3) outputs. What enters the products
//    besides the bf16 projections (decays, step sizes, the carried state) is fp32 split into two bf16 terms, so that nothing
//    of the recurrence is rounded to 8 bits of mantissa;
//  * step: one token per sequence, convolution included, for decoding.
//
// The convolution keeps its inputs in a ring of `taps` rows indexed by position: the row a token writes is never one that is
// read for it, so all heads of a group can read the shared B / C channels while one of them stores.
#include "hybrid.h"
#include "hybrid_common.cuh"

namespace mb {
namespace {

using namespace hy;

// exp(x) S for x <= 0 as fma(c, S, k S). A slow decay multiplies thousands of times, so that a bias of the rounded factor
// would add up; near 1 the factor is therefore applied as S + (exp(x) - 1) S.
struct Decay {
  float c, k;
  __device__ __forceinline__ explicit Decay(float x) {
    const bool near_one = x > -0.35f;
    c = near_one ? expm1f(x) : expf(x);
    k = near_one ? 1.f : 0.f;
  }
  __device__ __forceinline__ float operator()(float s) const { return fmaf(c, s, k * s); }
};

// ------------------------------------------------------------------------------------------------ convolution (prefill)
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) conv_kernel(const HyMamba a, const int4* __restrict__ tiles, T* __restrict__ xbc) {
  const int4 tl = tiles[blockIdx.x];
  const int inner = a.heads * a.P, ch = inner + 2 * a.groups * a.N;
  const int c = blockIdx.y * 128 + threadIdx.x;
  if (c >= ch) return;
  const int taps = TAPS > 0 ? TAPS : a.taps;
  const int seq = tl.x, row0 = tl.y, n = tl.z;
  const int first = a.cu[seq], ctx = a.ctx[seq];
  const long long slot = a.slots[seq];
  const T* in = static_cast<const T*>(a.proj) + inner + c;
  const T* ring = static_cast<const T*>(a.ring) + slot * taps * ch + c;
  const T* w = static_cast<const T*>(a.conv_w) + static_cast<long long>(c) * taps;
  const float bias = to_f(static_cast<const T*>(a.conv_b)[c]);
  // input of the token `back` rows before row r
  auto input = [&](int r, int back) -> float {
    const int q = r - back;
    if (q >= first) return to_f(in[static_cast<long long>(q) * a.ld]);
    const int p = ctx + q - first;
    return p < 0 ? 0.f : to_f(ring[static_cast<long long>(p % taps) * ch]);
  };
  if constexpr (TAPS > 0) {
    float wv[TAPS], hist[TAPS];
#pragma unroll
    for (int k = 0; k < TAPS; ++k) {
      wv[k] = to_f(w[k]);
      hist[k] = k + 1 < TAPS ? input(row0, TAPS - 1 - k) : 0.f;
    }
    for (int t = 0; t < n; ++t) {
      hist[TAPS - 1] = to_f(in[static_cast<long long>(row0 + t) * a.ld]);
      float v = bias;
#pragma unroll
      for (int k = 0; k < TAPS; ++k) v += wv[k] * hist[k];
#pragma unroll
      for (int k = 0; k + 1 < TAPS; ++k) hist[k] = hist[k + 1];
      xbc[static_cast<long long>(row0 + t) * ch + c] = from_f<T>(silu_f(v));
    }
  } else {
    for (int t = 0; t < n; ++t) {
      float v = bias;
      for (int k = 0; k < taps; ++k) v += to_f(w[k]) * input(row0 + t, taps - 1 - k);
      xbc[static_cast<long long>(row0 + t) * ch + c] = from_f<T>(silu_f(v));
    }
  }
}

// Two channels per thread for bf16 rows whose columns start on even offsets, four taps.
__global__ void __launch_bounds__(128) conv4_pair_kernel(const HyMamba a, const int4* __restrict__ tiles, bf16* __restrict__ xbc) {
  const int4 tl = tiles[blockIdx.x];
  const int inner = a.heads * a.P, ch = inner + 2 * a.groups * a.N;
  const int c = (blockIdx.y * 128 + threadIdx.x) * 2;
  if (c >= ch) return;
  const int seq = tl.x, row0 = tl.y, n = tl.z;
  const int first = a.cu[seq], ctx = a.ctx[seq];
  const bf16* in = static_cast<const bf16*>(a.proj) + inner + c;
  const bf16* ring = static_cast<const bf16*>(a.ring) + static_cast<long long>(a.slots[seq]) * 4 * ch + c;
  auto ld2 = [](const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); };
  auto input = [&](int r, int back) -> float2 {
    const int q = r - back;
    if (q >= first) return ld2(in + static_cast<long long>(q) * a.ld);
    const int p = ctx + q - first;
    return p < 0 ? make_float2(0.f, 0.f) : ld2(ring + static_cast<long long>(p & 3) * ch);
  };
  const bf16* w = static_cast<const bf16*>(a.conv_w) + static_cast<long long>(c) * 4;
  float2 wv[4], h0 = input(row0, 3), h1 = input(row0, 2), h2 = input(row0, 1);
#pragma unroll
  for (int k = 0; k < 4; ++k) wv[k] = make_float2(to_f(w[k]), to_f(w[4 + k]));
  const float2 bias = ld2(static_cast<const bf16*>(a.conv_b) + c);
#pragma unroll 4
  for (int t = 0; t < n; ++t) {
    const float2 h3 = ld2(in + static_cast<long long>(row0 + t) * a.ld);
    float x = bias.x, y = bias.y;
    x += wv[0].x * h0.x; y += wv[0].y * h0.y;
    x += wv[1].x * h1.x; y += wv[1].y * h1.y;
    x += wv[2].x * h2.x; y += wv[2].y * h2.y;
    x += wv[3].x * h3.x; y += wv[3].y * h3.y;
    h0 = h1; h1 = h2; h2 = h3;
    *reinterpret_cast<__nv_bfloat162*>(xbc + static_cast<long long>(row0 + t) * ch + c) = __floats2bfloat162_rn(silu_f(x), silu_f(y));
  }
}

// The last `taps` inputs of every sequence into its ring (after the convolution has read what was there).
template <typename T>
__global__ void __launch_bounds__(256) ring_kernel(const HyMamba a) {
  const int seq = blockIdx.x, inner = a.heads * a.P, ch = inner + 2 * a.groups * a.N;
  const int c = blockIdx.y * 256 + threadIdx.x;
  if (c >= ch) return;
  const int first = a.cu[seq], n = a.cu[seq + 1] - first, ctx = a.ctx[seq];
  const T* in = static_cast<const T*>(a.proj) + inner + c;
  T* ring = static_cast<T*>(a.ring) + static_cast<long long>(a.slots[seq]) * a.taps * ch + c;
  for (int q = max(0, n - a.taps); q < n; ++q)
    ring[static_cast<long long>((ctx + q) % a.taps) * ch] = in[static_cast<long long>(first + q) * a.ld];
}

// ------------------------------------------------------------------------------------------------ sequential scan
// One warp per state row p: lane l holds N values l, l + 32, ...
template <typename T, int NR>
__global__ void __launch_bounds__(256) scan_kernel(const HyMamba a, const T* __restrict__ xbc, T* __restrict__ y) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p = blockIdx.x * 8 + warp, h = blockIdx.y, seq = blockIdx.z;
  if (p >= a.P) return;
  const int inner = a.heads * a.P, ch = inner + 2 * a.groups * a.N, g = h / (a.heads / a.groups);
  const int first = a.cu[seq], n = a.cu[seq + 1] - first;
  float* st = a.state + ((static_cast<long long>(a.slots[seq]) * a.heads + h) * a.P + p) * a.N;
  float S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) S[i] = (a.ctx[seq] > 0 && lane + 32 * i < a.N) ? st[lane + 32 * i] : 0.f;
  const float A = -expf(to_f(static_cast<const T*>(a.A_log)[h])), D = to_f(static_cast<const T*>(a.D)[h]);
  const float bias = to_f(static_cast<const T*>(a.dt_bias)[h]);
  const T* dtc = static_cast<const T*>(a.proj) + inner + ch + h;
  for (int t = 0; t < n; ++t) {
    const long long r = first + t;
    const T* row = xbc + r * ch;
    const float dt = softplus_f(to_f(dtc[r * a.ld]) + bias);
    const Decay decay(A * dt);
    const float x = to_f(row[h * a.P + p]);
    const T *B = row + inner + g * a.N, *C = B + a.groups * a.N;
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int k = lane + 32 * i;
      if (k < a.N) {
        S[i] = decay(S[i]) + dt * to_f(B[k]) * x;
        o += S[i] * to_f(C[k]);
      }
    }
    o = warp_sum(o);
    if (lane == 0) y[r * inner + h * a.P + p] = from_f<T>(o + D * x);
  }
#pragma unroll
  for (int i = 0; i < NR; ++i)
    if (lane + 32 * i < a.N) st[lane + 32 * i] = S[i];
}

// ------------------------------------------------------------------------------------------------ one token
// CTA = (head, sequence). Convolution of the head's own channels and its group's B / C, then the state update; a warp walks
// the rows p, VEC4: every lane owns 4 consecutive values of a 128-wide block of N.
template <typename T, bool VEC4>
__global__ void __launch_bounds__(256) step_kernel(const HyMamba a, const int* __restrict__ positions, T* __restrict__ y) {
  extern __shared__ float sm[];  // x[P] | B[N] | C[N]
  const int h = blockIdx.x, b = blockIdx.y, P = a.P, N = a.N, taps = a.taps;
  const int inner = a.heads * P, ch = inner + 2 * a.groups * N, per = a.heads / a.groups, g = h / per;
  const int pos = positions[b];
  const long long slot = a.slots[b];
  if (slot < 0 || slot >= a.sequences) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, 11);
    return;
  }
  const T* pr = static_cast<const T*>(a.proj) + static_cast<long long>(b) * a.ld;
  T* ring = static_cast<T*>(a.ring) + slot * taps * ch;
  for (int i = threadIdx.x; i < P + 2 * N; i += blockDim.x) {
    const int c = i < P ? h * P + i : (i < P + N ? inner + g * N + i - P : inner + a.groups * N + g * N + i - P - N);
    const T* w = static_cast<const T*>(a.conv_w) + static_cast<long long>(c) * taps;
    float v = to_f(static_cast<const T*>(a.conv_b)[c]);
    for (int k = 0; k + 1 < taps; ++k) {
      const int q = pos - (taps - 1 - k);
      if (q >= 0) v += to_f(w[k]) * to_f(ring[static_cast<long long>(q % taps) * ch + c]);
    }
    const T cur = pr[inner + c];
    v += to_f(w[taps - 1]) * to_f(cur);
    if (i < P || h == g * per) ring[static_cast<long long>(pos % taps) * ch + c] = cur;
    sm[i] = to_f(from_f<T>(silu_f(v)));
  }
  __syncthreads();
  const float A = -expf(to_f(static_cast<const T*>(a.A_log)[h])), D = to_f(static_cast<const T*>(a.D)[h]);
  const float dt = softplus_f(to_f(pr[inner + ch + h]) + to_f(static_cast<const T*>(a.dt_bias)[h]));
  const Decay decay(A * dt);
  const float *x = sm, *B = sm + P, *C = B + N;
  float* st = a.state + (slot * a.heads + h) * static_cast<long long>(P) * N;
  T* out = y + static_cast<long long>(b) * inner + h * P;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const bool fresh = pos <= 0;
  if constexpr (VEC4) {
    constexpr int U = 4;  // rows in flight per warp
    for (int p0 = warp * U; p0 < P; p0 += nw * U) {
      float o[U];
#pragma unroll
      for (int u = 0; u < U; ++u) o[u] = 0.f;
      for (int k = lane * 4; k < N; k += 128) {
        float4 s[U];
#pragma unroll
        for (int u = 0; u < U; ++u)
          s[u] = (!fresh && p0 + u < P) ? *reinterpret_cast<const float4*>(st + static_cast<long long>(p0 + u) * N + k) : make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 bv = *reinterpret_cast<const float4*>(B + k), cv = *reinterpret_cast<const float4*>(C + k);
#pragma unroll
        for (int u = 0; u < U; ++u) {
          if (p0 + u >= P) break;
          const float xp = x[p0 + u];
          s[u].x = decay(s[u].x) + dt * bv.x * xp;
          s[u].y = decay(s[u].y) + dt * bv.y * xp;
          s[u].z = decay(s[u].z) + dt * bv.z * xp;
          s[u].w = decay(s[u].w) + dt * bv.w * xp;
          o[u] += s[u].x * cv.x + s[u].y * cv.y + s[u].z * cv.z + s[u].w * cv.w;
          *reinterpret_cast<float4*>(st + static_cast<long long>(p0 + u) * N + k) = s[u];
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        o[u] = warp_sum(o[u]);
        if (lane == 0 && p0 + u < P) out[p0 + u] = from_f<T>(o[u] + D * x[p0 + u]);
      }
    }
  } else {
    for (int p = warp; p < P; p += nw) {
      float o = 0.f;
      float* row = st + static_cast<long long>(p) * N;
      for (int k = lane; k < N; k += 32) {
        const float s = decay(fresh ? 0.f : row[k]) + dt * B[k] * x[p];
        row[k] = s;
        o += s * C[k];
      }
      o = warp_sum(o);
      if (lane == 0) out[p] = from_f<T>(o + D * x[p]);
    }
  }
}

// ------------------------------------------------------------------------------------------------ chunked scan (bf16)
constexpr int Q = HY_CHUNK;      // tokens per chunk
constexpr int CW = 8;            // warps
constexpr int LDX_PAD = 8;       // bf16 elements added to shared rows: conflict-free ldmatrix

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

// dt and the running sum of -exp(A_log) dt over the chunk: smem dt[Q], acum[Q] (zeros past n keep the sum flat)
__device__ __forceinline__ void chunk_decay(const HyMamba& a, int h, int row0, int n, float* dts, float* acum) {
  const int inner = a.heads * a.P, ch = inner + 2 * a.groups * a.N;
  if (threadIdx.x < Q) {
    float dt = 0.f;
    if (static_cast<int>(threadIdx.x) < n)
      dt = softplus_f(to_f(static_cast<const bf16*>(a.proj)[static_cast<long long>(row0 + threadIdx.x) * a.ld + inner + ch + h]) +
                      to_f(static_cast<const bf16*>(a.dt_bias)[h]));
    dts[threadIdx.x] = dt;
    float v = -expf(to_f(static_cast<const bf16*>(a.A_log)[h])) * dt;
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float u = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= o) v += u;
    }
    acum[threadIdx.x] = v;
  }
  __syncthreads();
  float base = 0.f;
  if (threadIdx.x < Q)
    for (int w = 0; w < static_cast<int>(threadIdx.x >> 5); ++w) base += acum[w * 32 + 31];
  __syncthreads();
  if (threadIdx.x < Q) acum[threadIdx.x] += base;
  __syncthreads();
}

// rows [n, w] of xbc starting at column c0 into smem [Q][ld], zero filled to wp columns and Q rows
__device__ __forceinline__ void load_tile(const bf16* __restrict__ xbc, long long ch, int row0, int n, int c0, int w, int wp,
                                          bf16* dst, int ld, bool vec) {
  if (vec) {
    const int per = wp / 8;
    for (int i = threadIdx.x; i < Q * per; i += CW * 32) {
      const int r = i / per, c = (i - r * per) * 8;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < n && c < w) v = *reinterpret_cast<const uint4*>(xbc + (row0 + r) * ch + c0 + c);
      *reinterpret_cast<uint4*>(dst + r * ld + c) = v;
    }
  } else {
    for (int i = threadIdx.x; i < Q * wp; i += CW * 32) {
      const int r = i / wp, c = i - r * wp;
      dst[r * ld + c] = (r < n && c < w) ? xbc[(row0 + r) * ch + c0 + c] : __float2bfloat16(0.f);
    }
  }
}

// (1) work[chunk, h, p, n] = sum_t exp(acum_end - acum_t) dt_t x_t[p] B_t[n];  decay[chunk, h] = exp(acum_end)
__global__ void __launch_bounds__(CW * 32) chunk_state_kernel(const HyMamba a, const bf16* __restrict__ xbc,
                                                              const int4* __restrict__ chunks, float* __restrict__ work,
                                                              float* __restrict__ decay, bool vec) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int4 ck = chunks[blockIdx.x];
  const int h = blockIdx.y, row0 = ck.y, n = ck.z;
  const int P = a.P, N = a.N, PP = (P + 15) / 16 * 16, NP = (N + 63) / 64 * 64;
  const int inner = a.heads * P, ch = inner + 2 * a.groups * N, g = h / (a.heads / a.groups);
  const int ldx = PP + LDX_PAD, ldb = NP + LDX_PAD;
  bf16* xh = reinterpret_cast<bf16*>(raw);   // [Q][ldx] weighted x, high part
  bf16* xl = xh + Q * ldx;                   // low part
  bf16* Bs = xl + Q * ldx;                   // [Q][ldb]
  float* dts = reinterpret_cast<float*>(Bs + Q * ldb);
  float* acum = dts + Q;
  chunk_decay(a, h, row0, n, dts, acum);
  load_tile(xbc, ch, row0, n, inner + g * N, N, NP, Bs, ldb, vec);
  const float end = acum[Q - 1];
  for (int i = threadIdx.x; i < Q * (PP / 2); i += CW * 32) {
    const int r = i / (PP / 2), c = (i - r * (PP / 2)) * 2;
    float u = 0.f, v = 0.f;
    if (r < n) {
      const float w = expf(end - acum[r]) * dts[r];
      const bf16* src = xbc + static_cast<long long>(row0 + r) * ch + h * P + c;
      if (c < P) u = w * to_f(src[0]);
      if (c + 1 < P) v = w * to_f(src[1]);
    }
    uint32_t hi, lo;
    split2(u, v, hi, lo);
    *reinterpret_cast<uint32_t*>(xh + r * ldx + c) = hi;
    *reinterpret_cast<uint32_t*>(xl + r * ldx + c) = lo;
  }
  if (threadIdx.x == 0) decay[static_cast<long long>(blockIdx.x) * a.heads + h] = expf(end);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* out = work + (static_cast<long long>(blockIdx.x) * a.heads + h) * P * N;
  const int mt = PP / 16, nt = NP / 64;
  for (int unit = warp; unit < mt * nt; unit += CW) {
    const int m0 = (unit % mt) * 16, n0 = (unit / mt) * 64;
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    for (int k0 = 0; k0 < Q; k0 += 16) {
      if (k0 >= n) break;
      uint32_t ah[4], al[4];
      // A = (weighted x)^T: rows p, contraction t; stored [t][p], so transpose while loading
      const int ar = k0 + (lane & 7) + ((lane >> 4) << 3), ac = m0 + (((lane >> 3) & 1) << 3);
      ldsm4t(s_u32(xh + ar * ldx + ac), ah);
      ldsm4t(s_u32(xl + ar * ldx + ac), al);
#pragma unroll
      for (int jp = 0; jp < 4; ++jp) {
        uint32_t b[4];
        const int br = k0 + (lane & 7) + (((lane >> 3) & 1) << 3), bc = n0 + jp * 16 + ((lane >> 4) << 3);
        ldsm4t(s_u32(Bs + br * ldb + bc), b);
        mma(acc[2 * jp], ah, b[0], b[1]);
        mma(acc[2 * jp], al, b[0], b[1]);
        mma(acc[2 * jp + 1], ah, b[2], b[3]);
        mma(acc[2 * jp + 1], al, b[2], b[3]);
      }
    }
    const int p0 = m0 + (lane >> 2);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int c = n0 + j * 8 + (lane & 3) * 2;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int p = p0 + (e >> 1) * 8, cc = c + (e & 1);
        if (p < P && cc < N) out[static_cast<long long>(p) * N + cc] = acc[j][e];
      }
    }
  }
}

// (2) replace every chunk's contribution by the state before the chunk; leave the state after the last in the slot
__global__ void __launch_bounds__(256) chunk_pass_kernel(const HyMamba a, const int* __restrict__ first_chunk,
                                                         const float* __restrict__ decay, float* __restrict__ work) {
  const int h = blockIdx.y, seq = blockIdx.z;
  const long long size = static_cast<long long>(a.P) * a.N;
  const long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= size) return;
  float* st = a.state + (static_cast<long long>(a.slots[seq]) * a.heads + h) * size + i;
  float s = a.ctx[seq] > 0 ? *st : 0.f;
  const int c1 = first_chunk[seq + 1];
  int c = first_chunk[seq];
  constexpr int U = 8;
  for (; c + U <= c1; c += U) {  // loads of several chunks in flight
    float v[U], d[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      v[u] = work[(static_cast<long long>(c + u) * a.heads + h) * size + i];
      d[u] = decay[static_cast<long long>(c + u) * a.heads + h];
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      work[(static_cast<long long>(c + u) * a.heads + h) * size + i] = s;
      s = d[u] * s + v[u];
    }
  }
  for (; c < c1; ++c) {
    float* w = work + (static_cast<long long>(c) * a.heads + h) * size + i;
    const float v = *w;
    *w = s;
    s = decay[static_cast<long long>(c) * a.heads + h] * s + v;
  }
  *st = s;
}

// (3) y[t] = exp(acum_t) C_t S_before + sum_{s <= t} (C_t . B_s) exp(acum_t - acum_s) dt_s x_s + D x_t
template <int PT>  // 16-wide tiles of P
__global__ void __launch_bounds__(CW * 32) chunk_out_kernel(const HyMamba a, const bf16* __restrict__ xbc,
                                                            const int4* __restrict__ chunks, const float* __restrict__ work,
                                                            bf16* __restrict__ y, bool vec) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int4 ck = chunks[blockIdx.x];
  const int h = blockIdx.y, seq = ck.x, row0 = ck.y, n = ck.z;
  const int P = a.P, N = a.N, NP = (N + 15) / 16 * 16;
  const int inner = a.heads * P, ch = inner + 2 * a.groups * N, g = h / (a.heads / a.groups);
  constexpr int PP = PT * 16;
  constexpr int ldx = PP + LDX_PAD;
  const int ldn = NP + LDX_PAD;
  bf16* Cs = reinterpret_cast<bf16*>(raw);  // [Q][ldn]
  bf16* Bs = Cs + Q * ldn;                  // [Q][ldn]
  bf16* xs = Bs + Q * ldn;                  // [Q][ldx]
  bf16* Sh = xs + Q * ldx;                  // [PP][ldn] carried state, high part
  bf16* Sl = Sh + PP * ldn;                 // low part
  float* dts = reinterpret_cast<float*>(Sl + PP * ldn);
  float* acum = dts + Q;
  const bool carried = ck.w > 0 || a.ctx[seq] > 0;
  load_tile(xbc, ch, row0, n, inner + a.groups * N + g * N, N, NP, Cs, ldn, vec);
  load_tile(xbc, ch, row0, n, inner + g * N, N, NP, Bs, ldn, vec);
  load_tile(xbc, ch, row0, n, h * P, P, PP, xs, ldx, vec);
  if (carried) {
    const float* src = work + (static_cast<long long>(blockIdx.x) * a.heads + h) * P * N;
    for (int i = threadIdx.x; i < PP * (NP / 2); i += CW * 32) {
      const int p = i / (NP / 2), c = (i - p * (NP / 2)) * 2;
      float u = 0.f, v = 0.f;
      if (p < P) {
        if (c < N) u = src[static_cast<long long>(p) * N + c];
        if (c + 1 < N) v = src[static_cast<long long>(p) * N + c + 1];
      }
      uint32_t hi, lo;
      split2(u, v, hi, lo);
      *reinterpret_cast<uint32_t*>(Sh + p * ldn + c) = hi;
      *reinterpret_cast<uint32_t*>(Sl + p * ldn + c) = lo;
    }
  }
  chunk_decay(a, h, row0, n, dts, acum);  // ends with a block barrier
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = warp * 16;
  if (t0 >= n) return;
  const int r0 = t0 + (lane >> 2);  // this lane's rows: r0 and r0 + 8
  float o[2 * PT][4];
#pragma unroll
  for (int j = 0; j < 2 * PT; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  const int a_row = t0 + (lane & 15), a_col = (lane >> 4) << 3;
  if (carried) {
    for (int k0 = 0; k0 < NP; k0 += 16) {
      uint32_t cf[4];
      ldsm4(s_u32(Cs + a_row * ldn + k0 + a_col), cf);
#pragma unroll
      for (int jp = 0; jp < PT; ++jp) {
        uint32_t b[4];
        const int br = jp * 16 + (lane & 7) + ((lane >> 4) << 3), bc = k0 + (((lane >> 3) & 1) << 3);
        ldsm4(s_u32(Sh + br * ldn + bc), b);
        mma(o[2 * jp], cf, b[0], b[1]);
        mma(o[2 * jp + 1], cf, b[2], b[3]);
        ldsm4(s_u32(Sl + br * ldn + bc), b);
        mma(o[2 * jp], cf, b[0], b[1]);
        mma(o[2 * jp + 1], cf, b[2], b[3]);
      }
    }
    const float e0 = expf(acum[r0]), e1 = expf(acum[r0 + 8]);
#pragma unroll
    for (int j = 0; j < 2 * PT; ++j) {
      o[j][0] *= e0; o[j][1] *= e0;
      o[j][2] *= e1; o[j][3] *= e1;
    }
  }
  const float ac0 = acum[r0], ac1 = acum[r0 + 8];
  for (int s0 = 0; s0 <= t0; s0 += 16) {  // blocks of 16 earlier tokens
    float sc[2][4];
    sc[0][0] = sc[0][1] = sc[0][2] = sc[0][3] = 0.f;
    sc[1][0] = sc[1][1] = sc[1][2] = sc[1][3] = 0.f;
    for (int k0 = 0; k0 < NP; k0 += 16) {
      uint32_t cf[4], b[4];
      ldsm4(s_u32(Cs + a_row * ldn + k0 + a_col), cf);
      ldsm4(s_u32(Bs + (s0 + (lane & 7) + ((lane >> 4) << 3)) * ldn + k0 + (((lane >> 3) & 1) << 3)), b);
      mma(sc[0], cf, b[0], b[1]);
      mma(sc[1], cf, b[2], b[3]);
    }
    // scores -> decay-weighted coefficients, split in two bf16 terms; accumulator layout = A-operand layout
    uint32_t wh[4], wl[4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      float w[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int s = s0 + nt * 8 + (lane & 3) * 2 + (e & 1), t = r0 + (e >> 1) * 8;
        w[e] = s <= t ? sc[nt][e] * expf((e >> 1 ? ac1 : ac0) - acum[s]) * dts[s] : 0.f;
      }
      split2(w[0], w[1], wh[nt * 2], wl[nt * 2]);
      split2(w[2], w[3], wh[nt * 2 + 1], wl[nt * 2 + 1]);
    }
#pragma unroll
    for (int jp = 0; jp < PT; ++jp) {
      uint32_t b[4];
      ldsm4t(s_u32(xs + (s0 + (lane & 7) + (((lane >> 3) & 1) << 3)) * ldx + jp * 16 + ((lane >> 4) << 3)), b);
      mma(o[2 * jp], wh, b[0], b[1]);
      mma(o[2 * jp], wl, b[0], b[1]);
      mma(o[2 * jp + 1], wh, b[2], b[3]);
      mma(o[2 * jp + 1], wl, b[2], b[3]);
    }
  }
  const float D = to_f(static_cast<const bf16*>(a.D)[h]);
#pragma unroll
  for (int j = 0; j < 2 * PT; ++j) {
    const int p = j * 8 + (lane & 3) * 2;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = r0 + e * 8;
      if (t >= n) continue;
      bf16* dst = y + static_cast<long long>(row0 + t) * inner + h * P + p;
      const float u = o[j][2 * e] + D * to_f(xs[t * ldx + p]), v = o[j][2 * e + 1] + D * to_f(xs[t * ldx + p + 1]);
      if (p + 1 < P && (P & 1) == 0) {
        *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(u, v);
      } else {
        if (p < P) dst[0] = __float2bfloat16(u);
        if (p + 1 < P) dst[1] = __float2bfloat16(v);
      }
    }
  }
}

template <typename T>
int conv_t(const HyMamba& a, const int* tiles, int n_tiles, void* xbc, cudaStream_t s) {
  const int ch = a.heads * a.P + 2 * a.groups * a.N;
  const int4* tl = reinterpret_cast<const int4*>(tiles);
  const dim3 grid(n_tiles, (ch + 127) / 128);
  T* out = static_cast<T*>(xbc);
  bool done = false;
  if constexpr (sizeof(T) == 2) {
    if (a.taps == 4 && (a.heads * a.P) % 2 == 0 && ch % 2 == 0 && a.ld % 2 == 0) {
      conv4_pair_kernel<<<dim3(n_tiles, (ch + 255) / 256), 128, 0, s>>>(a, tl, out);
      done = true;
    }
  }
  if (!done) {
    switch (a.taps) {
      case 2: conv_kernel<T, 2><<<grid, 128, 0, s>>>(a, tl, out); break;
      case 3: conv_kernel<T, 3><<<grid, 128, 0, s>>>(a, tl, out); break;
      case 4: conv_kernel<T, 4><<<grid, 128, 0, s>>>(a, tl, out); break;
      default: conv_kernel<T, 0><<<grid, 128, 0, s>>>(a, tl, out); break;
    }
  }
  ring_kernel<T><<<dim3(a.nseq, (ch + 255) / 256), 256, 0, s>>>(a);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int scan_t(const HyMamba& a, const void* xbc, void* y, cudaStream_t s) {
  const dim3 grid((a.P + 7) / 8, a.heads, a.nseq);
  const T* in = static_cast<const T*>(xbc);
  T* out = static_cast<T*>(y);
  if (a.N <= 32) scan_kernel<T, 1><<<grid, 256, 0, s>>>(a, in, out);
  else if (a.N <= 64) scan_kernel<T, 2><<<grid, 256, 0, s>>>(a, in, out);
  else if (a.N <= 128) scan_kernel<T, 4><<<grid, 256, 0, s>>>(a, in, out);
  else if (a.N <= 256) scan_kernel<T, 8><<<grid, 256, 0, s>>>(a, in, out);
  else if (a.N <= 1024) scan_kernel<T, 32><<<grid, 256, 0, s>>>(a, in, out);
  else return static_cast<int>(cudaErrorInvalidValue);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int step_t(const HyMamba& a, const int* positions, int B, void* y, cudaStream_t s) {
  const size_t smem = sizeof(float) * (static_cast<size_t>(a.P) + 2 * a.N);
  const bool vec = a.N % 4 == 0 && a.P % 4 == 0;
  auto kern = vec ? step_kernel<T, true> : step_kernel<T, false>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(a.heads, B), 256, smem, s>>>(a, positions, static_cast<T*>(y));
  return static_cast<int>(cudaGetLastError());
}

size_t state_smem(int P, int N) {
  const int PP = (P + 15) / 16 * 16, NP = (N + 63) / 64 * 64;
  return static_cast<size_t>(2) * (2 * Q * (PP + LDX_PAD) + Q * (NP + LDX_PAD)) + 2 * Q * sizeof(float);
}
size_t out_smem(int PP, int N) {
  const int NP = (N + 15) / 16 * 16;
  return static_cast<size_t>(2) * (2 * Q * (NP + LDX_PAD) + Q * (PP + LDX_PAD) + 2 * PP * (NP + LDX_PAD)) + 2 * Q * sizeof(float);
}
int out_tiles(int P) {
  const int t = (P + 15) / 16;
  return t <= 2 ? 2 : (t <= 3 ? 3 : (t <= 4 ? 4 : (t <= 6 ? 6 : 8)));
}

template <int PT>
int launch_out(const HyMamba& a, const bf16* xbc, const int4* ck, int n_chunks, const float* work, bf16* y, bool vec, cudaStream_t s) {
  const size_t smem = out_smem(PT * 16, a.N);
  auto kern = chunk_out_kernel<PT>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(n_chunks, a.heads), CW * 32, smem, s>>>(a, xbc, ck, work, y, vec);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace

int hy_conv(bool f32, const HyMamba& a, const int* tiles, int n_tiles, void* xbc, cudaStream_t s) {
  return f32 ? conv_t<float>(a, tiles, n_tiles, xbc, s) : conv_t<bf16>(a, tiles, n_tiles, xbc, s);
}
int hy_scan(bool f32, const HyMamba& a, const void* xbc, void* y, cudaStream_t s) {
  return f32 ? scan_t<float>(a, xbc, y, s) : scan_t<bf16>(a, xbc, y, s);
}
int hy_mamba_step(bool f32, const HyMamba& a, const int* positions, int B, void* y, cudaStream_t s) {
  return f32 ? step_t<float>(a, positions, B, y, s) : step_t<bf16>(a, positions, B, y, s);
}

bool hy_chunk_scan_supported(int P, int N, int, int) {
  if (P < 1 || P > 128 || N < 1 || N > 256) return false;
  return state_smem(P, N) <= 227 * 1024 && out_smem(out_tiles(P) * 16, N) <= 227 * 1024;
}

int hy_chunk_scan(const HyMamba& a, const void* xbc_, const int* chunks, int n_chunks, const int* first_chunk, float* work,
                  float* decay, void* y_, cudaStream_t s) {
  if (!hy_chunk_scan_supported(a.P, a.N, a.heads, a.groups)) return static_cast<int>(cudaErrorInvalidValue);
  const bf16* xbc = static_cast<const bf16*>(xbc_);
  bf16* y = static_cast<bf16*>(y_);
  const int4* ck = reinterpret_cast<const int4*>(chunks);
  const bool vec = a.P % 8 == 0 && a.N % 8 == 0 && (reinterpret_cast<uintptr_t>(xbc) & 15) == 0;
  const size_t sm1 = state_smem(a.P, a.N);
  cudaError_t e = cudaFuncSetAttribute(chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(sm1));
  if (e != cudaSuccess) return static_cast<int>(e);
  chunk_state_kernel<<<dim3(n_chunks, a.heads), CW * 32, sm1, s>>>(a, xbc, ck, work, decay, vec);
  const long long size = static_cast<long long>(a.P) * a.N;
  chunk_pass_kernel<<<dim3(static_cast<unsigned>((size + 255) / 256), a.heads, a.nseq), 256, 0, s>>>(a, first_chunk, decay, work);
  e = cudaGetLastError();
  if (e != cudaSuccess) return static_cast<int>(e);
  switch (out_tiles(a.P)) {
    case 2: return launch_out<2>(a, xbc, ck, n_chunks, work, y, vec, s);
    case 3: return launch_out<3>(a, xbc, ck, n_chunks, work, y, vec, s);
    case 4: return launch_out<4>(a, xbc, ck, n_chunks, work, y, vec, s);
    case 6: return launch_out<6>(a, xbc, ck, n_chunks, work, y, vec, s);
    default: return launch_out<8>(a, xbc, ck, n_chunks, work, y, vec, s);
  }
}

}  // namespace mb
