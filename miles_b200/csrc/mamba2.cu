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
#include "hybrid_mma.cuh"

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

__device__ __forceinline__ long long state_row(const HyMamba& a, int seq) { return hy::state_row(a.slots, a.sequences, seq, a.status); }

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
  const long long slot = state_row(a, seq);
  const T* in = static_cast<const T*>(a.proj) + inner + c;
  const T* ring = static_cast<const T*>(a.ring) + (slot < 0 ? 0 : slot) * taps * ch + c;
  const T* w = static_cast<const T*>(a.conv_w) + static_cast<long long>(c) * taps;
  const float bias = to_f(static_cast<const T*>(a.conv_b)[c]);
  // input of the token `back` rows before row r
  auto input = [&](int r, int back) -> float {
    const int q = r - back;
    if (q >= first) return to_f(in[static_cast<long long>(q) * a.ld]);
    const int p = ctx + q - first;
    return p < 0 || slot < 0 ? 0.f : to_f(ring[static_cast<long long>(p % taps) * ch]);
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

// Eight channels per thread for bf16 rows whose columns start on 16-byte boundaries, four taps.
__global__ void __launch_bounds__(128) conv4_vec_kernel(const HyMamba a, const int4* __restrict__ tiles, bf16* __restrict__ xbc) {
  const int4 tl = tiles[blockIdx.x];
  const int inner = a.heads * a.P, ch = inner + 2 * a.groups * a.N;
  const int c = (blockIdx.y * 128 + threadIdx.x) * 8;
  if (c >= ch) return;
  const int seq = tl.x, row0 = tl.y, n = tl.z;
  const int first = a.cu[seq], ctx = a.ctx[seq];
  const bf16* in = static_cast<const bf16*>(a.proj) + inner + c;
  const long long slot = state_row(a, seq);
  const bf16* ring = static_cast<const bf16*>(a.ring) + (slot < 0 ? 0 : slot) * 4 * ch + c;
  float w[4][8], bias[8], h[3][8];
  {
    const bf16* wp = static_cast<const bf16*>(a.conv_w) + static_cast<long long>(c) * 4;  // [channel][tap]
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      float t[8];
      Vec<bf16>::load(wp + k * 8, t);  // channels 2k, 2k + 1
#pragma unroll
      for (int j = 0; j < 8; ++j) w[j & 3][2 * k + (j >> 2)] = t[j];
    }
  }
  Vec<bf16>::load(static_cast<const bf16*>(a.conv_b) + c, bias);
#pragma unroll
  for (int k = 0; k < 3; ++k) {  // inputs of the three tokens before the tile
    const int q = row0 - 3 + k, p = ctx + q - first;
    if (q >= first)
      Vec<bf16>::load(in + static_cast<long long>(q) * a.ld, h[k]);
    else if (p >= 0 && slot >= 0)
      Vec<bf16>::load(ring + static_cast<long long>(p & 3) * ch, h[k]);
    else
#pragma unroll
      for (int j = 0; j < 8; ++j) h[k][j] = 0.f;
  }
  constexpr int U = 4;  // tokens whose loads are in flight
  for (int t0 = 0; t0 < n; t0 += U) {
    uint4 raw[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (t0 + u < n) raw[u] = *reinterpret_cast<const uint4*>(in + static_cast<long long>(row0 + t0 + u) * a.ld);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (t0 + u >= n) break;
      const uint32_t r[4] = {raw[u].x, raw[u].y, raw[u].z, raw[u].w};
      float o[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r[j >> 1]));
        const float x = (j & 1) ? f.y : f.x;
        const float v = bias[j] + w[0][j] * h[0][j] + w[1][j] * h[1][j] + w[2][j] * h[2][j] + w[3][j] * x;
        h[0][j] = h[1][j];
        h[1][j] = h[2][j];
        h[2][j] = x;
        o[j] = __fdividef(v, 1.f + __expf(-v));
      }
      Vec<bf16>::store(xbc + static_cast<long long>(row0 + t0 + u) * ch + c, o);
    }
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
  const long long slot = state_row(a, seq);
  if (slot < 0) return;
  T* ring = static_cast<T*>(a.ring) + slot * a.taps * ch + c;
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
  const long long slot = state_row(a, seq);
  float* st = a.state + (((slot < 0 ? 0 : slot) * a.heads + h) * a.P + p) * a.N;
  float S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) S[i] = (slot >= 0 && a.ctx[seq] > 0 && lane + 32 * i < a.N) ? st[lane + 32 * i] : 0.f;
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
  if (slot < 0) return;
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

constexpr int MAX_HB = 8;        // heads of one group a CTA works on (a warp computes the decays of each)

// Warp w, head h0 + w, in units of log2: acum = running sum of -exp(A_log) dt over the chunk, src = acum - log2(dt), so that what
// token s hands to token t is exp2(acum_t - src_s) = exp(..) dt_s. Tokens past n get dt = 0: the sum stays flat, src = +inf. With
// log2_decay every token decays the state of head h by that much and dt = 1.
__device__ __forceinline__ void chunk_decays(const HyMamba& a, int h0, int nh, int row0, int n, float* src, float* acum) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp >= nh) return;
  const int h = h0 + warp, inner = a.heads * a.P, ch = inner + 2 * a.groups * a.N;
  float dt[Q / 32], v[Q / 32], run = 0.f;
  if (a.log2_decay) {
    const float A = a.log2_decay[h];
#pragma unroll
    for (int i = 0; i < Q / 32; ++i) {
      dt[i] = lane * (Q / 32) + i < n ? 1.f : 0.f;
      run += A * dt[i];
      v[i] = run;
    }
  } else {
    const bf16* col = static_cast<const bf16*>(a.proj) + inner + ch + h;
    const float bias = to_f(static_cast<const bf16*>(a.dt_bias)[h]), A = -expf(to_f(static_cast<const bf16*>(a.A_log)[h])) * LOG2E;
#pragma unroll
    for (int i = 0; i < Q / 32; ++i) {
      const int t = lane * (Q / 32) + i;
      dt[i] = t < n ? softplus_f(to_f(col[static_cast<long long>(row0 + t) * a.ld]) + bias) : 0.f;
      run += A * dt[i];
      v[i] = run;
    }
  }
  float base = run;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float u = __shfl_up_sync(0xffffffffu, base, o);
    if (lane >= o) base += u;
  }
  base -= run;
#pragma unroll
  for (int i = 0; i < Q / 32; ++i) {
    src[warp * Q + lane * (Q / 32) + i] = base + v[i] - log2f(dt[i]);
    acum[warp * Q + lane * (Q / 32) + i] = base + v[i];
  }
}

// (1) work[chunk, h, p, n] = sum_t exp(acum_end - acum_t) dt_t x_t[p] B_t[n];  decay[chunk, h] = exp(acum_end). A CTA takes
// several heads of a group: their B is the same tile.
template <int PT>
__global__ void __launch_bounds__(CW * 32, 2) chunk_state_kernel(const HyMamba a, const bf16* __restrict__ xbc,
                                                                 const int4* __restrict__ chunks, int hb, float* __restrict__ work,
                                                                 float* __restrict__ decay, bool vec) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int4 ck = chunks[blockIdx.x];
  const int row0 = ck.y, n = ck.z;
  const int P = a.P, N = a.N, NP = (N + 63) / 64 * 64, hpg = a.heads / a.groups;
  constexpr int PP = PT * 16, ldx = PP + LDX_PAD, XV = PP * Q / 8 / (CW * 32);
  const int per_group = (hpg + hb - 1) / hb, g = blockIdx.y / per_group;
  const int h0 = g * hpg + (blockIdx.y - g * per_group) * hb, nh = min(hb, (g + 1) * hpg - h0);
  const int ldb = NP + LDX_PAD;
  bf16* xh = reinterpret_cast<bf16*>(raw);   // [Q][ldx] weighted x, high part
  bf16* xl = xh + Q * ldx;                   // low part
  bf16* Bs = xl + Q * ldx;                   // [Q][ldb]
  float* srcs = reinterpret_cast<float*>(Bs + Q * ldb);  // [MAX_HB][Q]
  float* acum = srcs + MAX_HB * Q;
  load_tile<CW * 32>(xbc + row0 * a.xld + a.b_col + g * N, a.xld, n, N, Q, NP, Bs, ldb, vec);
  uint4 xr[XV];
  auto fetch = [&](int h) {
#pragma unroll
    for (int i = 0; i < XV; ++i) {
      const int k = threadIdx.x + i * CW * 32, r = k / (PP / 8), c = (k - r * (PP / 8)) * 8;
      xr[i] = make_uint4(0u, 0u, 0u, 0u);
      if (r >= n || c >= P) continue;
      const bf16* src = xbc + (row0 + r) * a.xld + a.x_col + h * P + c;
      if (vec) {
        xr[i] = *reinterpret_cast<const uint4*>(src);
      } else {
        bf16 t[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) t[j] = c + j < P ? src[j] : __float2bfloat16(0.f);
        xr[i] = *reinterpret_cast<const uint4*>(t);
      }
    }
  };
  fetch(h0);
  chunk_decays(a, h0, nh, row0, n, srcs, acum);
  cp_wait_all();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nt = NP / 64;
  for (int hi = 0; hi < nh; ++hi) {
    const int h = h0 + hi;
    const float* from = srcs + hi * Q;
    const float end = acum[hi * Q + Q - 1];
#pragma unroll
    for (int i = 0; i < XV; ++i) {
      const int k = threadIdx.x + i * CW * 32, r = k / (PP / 8), c = (k - r * (PP / 8)) * 8;
      const float w = ex2(end - from[r]);
      const uint32_t* q = reinterpret_cast<const uint32_t*>(&xr[i]);
      uint32_t hi4[4], lo4[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q[j]));
        split2(w * f.x, w * f.y, hi4[j], lo4[j]);
      }
      *reinterpret_cast<uint4*>(xh + r * ldx + c) = make_uint4(hi4[0], hi4[1], hi4[2], hi4[3]);
      *reinterpret_cast<uint4*>(xl + r * ldx + c) = make_uint4(lo4[0], lo4[1], lo4[2], lo4[3]);
    }
    if (hi + 1 < nh) fetch(h + 1);
    if (threadIdx.x == 0) decay[static_cast<long long>(blockIdx.x) * a.heads + h] = ex2(end);
    __syncthreads();
    float* out = work + (static_cast<long long>(blockIdx.x) * a.heads + h) * P * N;
    for (int unit = warp; unit < PT * nt; unit += CW) {
      const int m0 = (unit % PT) * 16, n0 = (unit / PT) * 64;
      float acc[8][4];
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll 2
      for (int k0 = 0; k0 < n; k0 += 16) {
        uint32_t ah[4], al[4];
        // A = (weighted x)^T: rows p, contraction t; stored [t][p], so transpose while loading
        const int ar = k0 + (lane & 7) + ((lane >> 4) << 3), acol = m0 + (((lane >> 3) & 1) << 3);
        ldsm4t(s_u32(xh + ar * ldx + acol), ah);
        ldsm4t(s_u32(xl + ar * ldx + acol), al);
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
        for (int e = 0; e < 2; ++e) {
          const int p = p0 + e * 8;
          if (p >= P) continue;
          float* dst = out + static_cast<long long>(p) * N + c;
          if ((N & 1) == 0) {
            if (c < N) *reinterpret_cast<float2*>(dst) = make_float2(acc[j][2 * e], acc[j][2 * e + 1]);
          } else {
            if (c < N) dst[0] = acc[j][2 * e];
            if (c + 1 < N) dst[1] = acc[j][2 * e + 1];
          }
        }
      }
    }
    __syncthreads();
  }
}

// (2) the state before every chunk, as two bf16 planes (high part, low part) [chunk, h, 2, P, N]; the state after the last chunk
// goes to the sequence's row. Decays are one per head, or (COLS) [chunk, h, 2, N]: one per column n, and a factor the planes are
// multiplied by
template <int V, bool COLS>
__global__ void __launch_bounds__(256) chunk_pass_kernel(const HyMamba a, const int* __restrict__ first_chunk,
                                                         const float* __restrict__ decay, const float* __restrict__ work,
                                                         bf16* __restrict__ before) {
  const int h = blockIdx.y, seq = blockIdx.z;
  const long long size = static_cast<long long>(a.P) * a.N;
  const long long i = (static_cast<long long>(blockIdx.x) * 256 + threadIdx.x) * V;
  if (i >= size) return;
  const long long slot = state_row(a, seq);
  float* st = a.state + ((slot < 0 ? 0 : slot) * a.heads + h) * size + i;
  float s[V];
  const bool cont = slot >= 0 && a.ctx[seq] > 0;
  auto load = [](const float* p, auto& v) {
    if constexpr (V == 4) {
      const float4 t = *reinterpret_cast<const float4*>(p);
      v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    } else {
      v[0] = p[0];
    }
  };
#pragma unroll
  for (int k = 0; k < V; ++k) s[k] = 0.f;
  if (cont) load(st, s);
  const int c0 = first_chunk[seq], c1 = first_chunk[seq + 1];
  constexpr int U = COLS ? 4 : 8;  // loads of several chunks in flight
  const int col = COLS ? static_cast<int>(i % a.N) : 0;
  for (int c = c0; c < c1; c += U) {
    float v[U][V], d[U][COLS ? V : 1], f[U][COLS ? V : 1];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c + u >= c1) break;
      const long long at = static_cast<long long>(c + u) * a.heads + h;
      load(work + at * size + i, v[u]);
      if constexpr (COLS) {
        load(decay + at * 2 * a.N + col, d[u]);
        load(decay + (at * 2 + 1) * a.N + col, f[u]);
      } else {
        d[u][0] = decay[at];
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (c + u >= c1) break;
      bf16* dst = before + (static_cast<long long>(c + u) * a.heads + h) * 2 * size + i;
      float b[V];
#pragma unroll
      for (int k = 0; k < V; ++k) b[k] = COLS ? s[k] * f[u][COLS ? k : 0] : s[k];
      if constexpr (V == 4) {
        uint32_t hi[2], lo[2];
        split2(b[0], b[1], hi[0], lo[0]);
        split2(b[2], b[3], hi[1], lo[1]);
        *reinterpret_cast<uint2*>(dst) = make_uint2(hi[0], hi[1]);
        *reinterpret_cast<uint2*>(dst + size) = make_uint2(lo[0], lo[1]);
      } else {
        const bf16 top = __float2bfloat16(b[0]);
        dst[0] = top;
        dst[size] = __float2bfloat16(b[0] - to_f(top));
      }
#pragma unroll
      for (int k = 0; k < V; ++k) s[k] = d[u][COLS ? k : 0] * s[k] + v[u][k];
    }
  }
  if (slot < 0) return;
  if constexpr (V == 4)
    *reinterpret_cast<float4*>(st) = make_float4(s[0], s[1], s[2], s[3]);
  else
    *st = s[0];
}

// (3) y[t] = exp(acum_t) C_t S_before + sum_{s <= t} (C_t . B_s) exp(acum_t - acum_s) dt_s x_s + D x_t
//
// A CTA takes several heads of a group: the products C B^T of the chunk are the same for all of them and are kept in shared
// memory, fragment by fragment. The lower triangle has 36 blocks of 16 x 16 tokens; a warp takes the row tiles (w, 7 - w), nine
// blocks, and 16 * PH columns p. With NBUF = 2 the next head's x and carried state arrive while this one computes.
constexpr int OW = 16;  // warps

template <int PH, int NBUF>
__global__ void __launch_bounds__(OW * 32, 1)
chunk_out_kernel(const HyMamba a, const bf16* __restrict__ xbc, const int4* __restrict__ chunks, int hb,
                 const bf16* __restrict__ before, bf16* __restrict__ y, bool vec) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int4 ck = chunks[blockIdx.x];
  const int seq = ck.x, row0 = ck.y, n = ck.z;
  const int P = a.P, N = a.N, NP = (N + 15) / 16 * 16, hpg = a.heads / a.groups;
  const int inner = a.heads * P;
  const int per_group = (hpg + hb - 1) / hb, g = blockIdx.y / per_group;
  const int h0 = g * hpg + (blockIdx.y - g * per_group) * hb, nh = min(hb, (g + 1) * hpg - h0);
  constexpr int PP = PH * 64;
  constexpr int ldx = PP + LDX_PAD;
  const int ldn = NP + LDX_PAD;
  float* Gs = reinterpret_cast<float*>(raw);             // [36][32 lanes][8]
  float* srcs = Gs + 36 * 256;                           // [MAX_HB][Q]
  float* acum = srcs + MAX_HB * Q;
  bf16* Cs = reinterpret_cast<bf16*>(acum + MAX_HB * Q); // [Q][ldn]
  bf16* xs = Cs + Q * ldn;                               // [NBUF][Q][ldx]
  bf16* Ss = xs + NBUF * Q * ldx;                        // [NBUF][2][PP][ldn]; the first one holds B before that
  const bool carried = ck.w > 0 || a.ctx[seq] > 0;
  const bf16* rows = xbc + row0 * a.xld;
  load_tile<OW * 32>(rows + a.c_col + g * N, a.xld, n, N, Q, NP, Cs, ldn, vec);
  load_tile<OW * 32>(rows + a.b_col + g * N, a.xld, n, N, Q, NP, Ss, ldn, vec);
  chunk_decays(a, h0, nh, row0, n, srcs, acum);
  cp_wait_all();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pg = warp >> 2, ta = warp & 3, tb = 7 - ta;     // column group, row tiles
  const int a_row = lane & 15, a_col = (lane >> 4) << 3;
  const int b_row = (lane & 7) + ((lane >> 4) << 3), b_col = ((lane >> 3) & 1) << 3;    // [n][k] operands
  const int v_row = (lane & 7) + (((lane >> 3) & 1) << 3), v_col = (lane >> 4) << 3;    // [k][n] operands
  for (int blk = warp; blk < 36; blk += OW) {
    int r = 0;
    while ((r + 1) * (r + 2) / 2 <= blk) ++r;
    const int s = blk - r * (r + 1) / 2;
    float g0[4] = {0.f, 0.f, 0.f, 0.f}, g1[4] = {0.f, 0.f, 0.f, 0.f};
    const uint32_t ca = s_u32(Cs + (r * 16 + a_row) * ldn + a_col), ba = s_u32(Ss + (s * 16 + b_row) * ldn + b_col);
#pragma unroll 4
    for (int k0 = 0; k0 < NP; k0 += 16) {
      uint32_t cf[4], b[4];
      ldsm4(ca + k0 * 2, cf);
      ldsm4(ba + k0 * 2, b);
      mma(g0, cf, b[0], b[1]);
      mma(g1, cf, b[2], b[3]);
    }
    float4* dst = reinterpret_cast<float4*>(Gs + blk * 256) + lane;  // two planes of 16 bytes per lane
    dst[0] = make_float4(g0[0], g0[1], g0[2], g0[3]);
    dst[32] = make_float4(g1[0], g1[1], g1[2], g1[3]);
  }
  __syncthreads();
  auto fetch = [&](int hi) {
    const int h = h0 + hi, buf = NBUF == 2 ? hi & 1 : 0;
    load_tile<OW * 32>(rows + a.x_col + h * P, a.xld, n, P, Q, PP, xs + buf * Q * ldx, ldx, vec);
    if (carried) {
      const bf16* src = before + (static_cast<long long>(blockIdx.x) * a.heads + h) * 2 * P * N;
      bf16* dst = Ss + buf * 2 * PP * ldn;
      load_tile<OW * 32>(src, N, P, N, PP, NP, dst, ldn, vec);
      load_tile<OW * 32>(src + static_cast<long long>(P) * N, N, P, N, PP, NP, dst + PP * ldn, ldn, vec);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);
  const int pc0 = pg * PH * 16;  // first column of this warp
  for (int hi = 0; hi < nh; ++hi) {
    const int h = h0 + hi, buf = NBUF == 2 ? hi & 1 : 0;
    if (NBUF == 2 && hi + 1 < nh) {
      fetch(hi + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    if (pc0 < P) {
      const bf16* xb = xs + buf * Q * ldx;
      const bf16* sb = Ss + buf * 2 * PP * ldn;
      const float* ac = acum + hi * Q;
      const float* from = srcs + hi * Q;
      const float D = a.D ? to_f(static_cast<const bf16*>(a.D)[h]) : 0.f;
#pragma unroll 1
      for (int half = 0; half < 2; ++half) {
        const int tile = half == 0 ? ta : tb;
        if (tile * 16 >= n) continue;
        const int r0 = tile * 16 + (lane >> 2);
        const float ac0 = ac[r0], ac1 = ac[r0 + 8];
        float o[2 * PH][4];
#pragma unroll
        for (int j = 0; j < 2 * PH; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
        if (carried) {  // what the carried state gives; the two parts of the split in accumulators of their own
          float q[2 * PH][4];
#pragma unroll
          for (int j = 0; j < 2 * PH; ++j) q[j][0] = q[j][1] = q[j][2] = q[j][3] = 0.f;
          const uint32_t ca = s_u32(Cs + (tile * 16 + a_row) * ldn + a_col), sa = s_u32(sb + (pc0 + b_row) * ldn + b_col);
#pragma unroll 4
          for (int k0 = 0; k0 < NP; k0 += 16) {
            uint32_t cf[4];
            ldsm4(ca + k0 * 2, cf);
#pragma unroll
            for (int jp = 0; jp < PH; ++jp) {
              uint32_t b[4], c[4];
              ldsm4(sa + (jp * 16 * ldn + k0) * 2, b);
              ldsm4(sa + ((PP + jp * 16) * ldn + k0) * 2, c);
              mma(o[2 * jp], cf, b[0], b[1]);
              mma(o[2 * jp + 1], cf, b[2], b[3]);
              mma(q[2 * jp], cf, c[0], c[1]);
              mma(q[2 * jp + 1], cf, c[2], c[3]);
            }
          }
          const float e0 = ex2(ac0), e1 = ex2(ac1);
#pragma unroll
          for (int j = 0; j < 2 * PH; ++j) {
            o[j][0] = (o[j][0] + q[j][0]) * e0; o[j][1] = (o[j][1] + q[j][1]) * e0;
            o[j][2] = (o[j][2] + q[j][2]) * e1; o[j][3] = (o[j][3] + q[j][3]) * e1;
          }
        }
        const float4* gp = reinterpret_cast<const float4*>(Gs + tile * (tile + 1) / 2 * 256) + lane;
        auto block = [&](int st, bool diag) {
          const int s0 = st * 16;
          // scores -> decay-weighted coefficients, split in two bf16 terms; accumulator layout = A-operand layout
          uint32_t wh[4], wl[4];
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            const int s = s0 + nt * 8 + (lane & 3) * 2;
            const float4 gv = gp[st * 64 + nt * 32];
            const float2 as = *reinterpret_cast<const float2*>(from + s);
            float w0 = gv.x * ex2(ac0 - as.x), w1 = gv.y * ex2(ac0 - as.y), w2 = gv.z * ex2(ac1 - as.x), w3 = gv.w * ex2(ac1 - as.y);
            if (diag) {  // only tokens up to t
              w0 = s <= r0 ? w0 : 0.f;
              w1 = s + 1 <= r0 ? w1 : 0.f;
              w2 = s <= r0 + 8 ? w2 : 0.f;
              w3 = s + 1 <= r0 + 8 ? w3 : 0.f;
            }
            split2(w0, w1, wh[nt * 2], wl[nt * 2]);
            split2(w2, w3, wh[nt * 2 + 1], wl[nt * 2 + 1]);
          }
          const uint32_t xa = s_u32(xb + (s0 + v_row) * ldx + pc0 + v_col);
#pragma unroll
          for (int jp = 0; jp < PH; ++jp) {
            uint32_t b[4];
            ldsm4t(xa + jp * 32, b);
            mma(o[2 * jp], wh, b[0], b[1]);
            mma(o[2 * jp + 1], wh, b[2], b[3]);
            mma(o[2 * jp], wl, b[0], b[1]);
            mma(o[2 * jp + 1], wl, b[2], b[3]);
          }
        };
#pragma unroll 2
        for (int st = 0; st < tile; ++st) block(st, false);
        block(tile, true);
#pragma unroll
        for (int j = 0; j < 2 * PH; ++j) {
          const int p = pc0 + j * 8 + (lane & 3) * 2;
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int t = r0 + e * 8;
            if (t >= n) continue;
            bf16* dst = y + static_cast<long long>(row0 + t) * inner + h * P + p;
            const float2 xv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(xb + t * ldx + p));
            const float u = o[j][2 * e] + D * xv.x, v = o[j][2 * e + 1] + D * xv.y;
            if ((P & 1) == 0) {
              if (p < P) *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(u, v);
            } else {
              if (p < P) dst[0] = __float2bfloat16(u);
              if (p + 1 < P) dst[1] = __float2bfloat16(v);
            }
          }
        }
      }
    }
    __syncthreads();  // this head's tiles have been read
    if (NBUF == 1 && hi + 1 < nh) fetch(hi + 1);
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
    if (a.taps == 4 && (a.heads * a.P) % 8 == 0 && ch % 8 == 0 && aligned16<T>(a.proj, a.ld) && aligned16<T>(a.ring, ch) &&
        aligned16<T>(a.conv_w, 8) && aligned16<T>(a.conv_b, 8)) {
      conv4_vec_kernel<<<dim3(n_tiles, (ch / 8 + 127) / 128), 128, 0, s>>>(a, tl, out);
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

size_t state_smem(int PT, int N) {
  const int NP = (N + 63) / 64 * 64;
  return static_cast<size_t>(2) * (2 * Q * (PT * 16 + LDX_PAD) + Q * (NP + LDX_PAD)) + 2 * MAX_HB * Q * sizeof(float);
}
size_t out_smem(int PH, int N, int nbuf) {
  const int NP = (N + 15) / 16 * 16, PP = PH * 64;
  return sizeof(float) * (36 * 256 + 2 * MAX_HB * Q) +
         static_cast<size_t>(2) * (Q * (NP + LDX_PAD) + nbuf * (Q * (PP + LDX_PAD) + 2 * PP * (NP + LDX_PAD)));
}
int half_tiles(int P) { return (P + 31) / 32; }

// heads per CTA: as many as leave the device a few waves of CTAs
int heads_per_cta(int n_chunks, int heads, int groups) {
  const int hpg = heads / groups;
  int hb = hpg < MAX_HB ? hpg : MAX_HB;
  while (hb > 1 && static_cast<long long>(n_chunks) * groups * ((hpg + hb - 1) / hb) < 3 * 2 * 148) hb = (hb + 1) / 2;
  return hb;
}

template <int PT>
int launch_state(const HyMamba& a, const bf16* xbc, const int4* ck, int n_chunks, int hb, float* work, float* decay, bool vec, cudaStream_t s) {
  const size_t smem = state_smem(PT, a.N);
  auto kern = chunk_state_kernel<PT>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  const int hpg = a.heads / a.groups;
  kern<<<dim3(n_chunks, a.groups * ((hpg + hb - 1) / hb)), CW * 32, smem, s>>>(a, xbc, ck, hb, work, decay, vec);
  return static_cast<int>(cudaGetLastError());
}

template <int PH, int NBUF>
int launch_out(const HyMamba& a, const bf16* xbc, const int4* ck, int n_chunks, int hb, const bf16* before, bf16* y, bool vec, cudaStream_t s) {
  const size_t smem = out_smem(PH, a.N, NBUF);
  auto kern = chunk_out_kernel<PH, NBUF>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  const int hpg = a.heads / a.groups;
  kern<<<dim3(n_chunks, a.groups * ((hpg + hb - 1) / hb)), OW * 32, smem, s>>>(a, xbc, ck, hb, before, y, vec);
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
  const int ph = half_tiles(P);
  return state_smem(2 * ph, N) <= 227 * 1024 && out_smem(P <= 64 ? 1 : 2, N, 1) <= 227 * 1024;
}

int hy_chunk_pass(const HyMamba& a, const int* first_chunk, const float* decay, bool cols, const float* work, void* before_, cudaStream_t s) {
  const long long size = static_cast<long long>(a.P) * a.N;
  bf16* before = static_cast<bf16*>(before_);
  const bool four = cols ? a.N % 4 == 0 : size % 4 == 0;
  const dim3 grid(static_cast<unsigned>(((four ? size / 4 : size) + 255) / 256), a.heads, a.nseq);
  if (four && cols) chunk_pass_kernel<4, true><<<grid, 256, 0, s>>>(a, first_chunk, decay, work, before);
  else if (four) chunk_pass_kernel<4, false><<<grid, 256, 0, s>>>(a, first_chunk, decay, work, before);
  else if (cols) chunk_pass_kernel<1, true><<<grid, 256, 0, s>>>(a, first_chunk, decay, work, before);
  else chunk_pass_kernel<1, false><<<grid, 256, 0, s>>>(a, first_chunk, decay, work, before);
  return static_cast<int>(cudaGetLastError());
}

int hy_chunk_scan(const HyMamba& a, const void* xbc_, const int* chunks, int n_chunks, const int* first_chunk, float* work,
                  float* decay, void* before_, void* y_, cudaStream_t s) {
  if (!hy_chunk_scan_supported(a.P, a.N, a.heads, a.groups)) return static_cast<int>(cudaErrorInvalidValue);
  const bf16* xbc = static_cast<const bf16*>(xbc_);
  bf16 *y = static_cast<bf16*>(y_), *before = static_cast<bf16*>(before_);
  const int4* ck = reinterpret_cast<const int4*>(chunks);
  const bool vec = a.P % 8 == 0 && a.N % 8 == 0 && (a.x_col | a.b_col | a.c_col) % 8 == 0 && aligned16<bf16>(xbc, a.xld);
  const int ph = half_tiles(a.P), hb = heads_per_cta(n_chunks, a.heads, a.groups);
  int rc = 0;
  switch (ph) {
    case 1: rc = launch_state<2>(a, xbc, ck, n_chunks, hb, work, decay, vec, s); break;
    case 2: rc = launch_state<4>(a, xbc, ck, n_chunks, hb, work, decay, vec, s); break;
    case 3: rc = launch_state<6>(a, xbc, ck, n_chunks, hb, work, decay, vec, s); break;
    default: rc = launch_state<8>(a, xbc, ck, n_chunks, hb, work, decay, vec, s); break;
  }
  if (rc != 0) return rc;
  rc = hy_chunk_pass(a, first_chunk, decay, false, work, before, s);
  if (rc != 0) return rc;
  const bool two = out_smem(a.P <= 64 ? 1 : 2, a.N, 2) <= 227 * 1024;
  if (a.P <= 64)
    return two ? launch_out<1, 2>(a, xbc, ck, n_chunks, hb, before, y, vec, s) : launch_out<1, 1>(a, xbc, ck, n_chunks, hb, before, y, vec, s);
  return two ? launch_out<2, 2>(a, xbc, ck, n_chunks, hb, before, y, vec, s) : launch_out<2, 1>(a, xbc, ck, n_chunks, hb, before, y, vec, s);
}

}  // namespace mb
