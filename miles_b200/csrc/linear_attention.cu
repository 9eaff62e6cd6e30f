// Linear attention with a decaying state: S <- S diag(a_t) + v_t k_t^T, o_t = S q_t, per head on a state [P, N] in fp32 (rows: values,
// columns: key channels). The decay a_t is a constant of the head, or one number per key channel and token, sigmoid(W2 u + b)^(1 / tau).
//
// Ways through the recurrence, as for Mamba-2 (whose chunked kernels serve constant decays: values are its x, keys its B, queries its C):
//  * scan: token after token, a warp per state row (any sizes, fp32 throughout);
//  * chunks with a decay per channel, 128 tokens at a time on the tensor cores. With c_t the running sum of log2 a over a chunk,
//        o_t = S_0 (q_t 2^c_t) + sum_{s <= t} (q_t . k_s 2^(c_t - c_s)) v_s
//    factors into products of q_t 2^(c_t - r) and k_s 2^(r - c_s) for a reference r per channel. One reference for the whole chunk (the
//    sums at its middle) serves as long as no channel moves by more than 2^+-60 from it. Chunks where one does take a reference per
//    16 tokens (both factors then stay below 1) and evaluate the blocks on the diagonal directly;
//  * step: one token per sequence, with rotation, decay, output norm and gate, for decoding.
// What enters the products besides the bf16 projections goes in as two bf16 terms (16 bits of mantissa), as does the carried state.
//
// Decays are applied as S + (a - 1) S with a - 1 from expm1: a slow decay multiplies thousands of times, and a rounded factor would
// drift.
#include <type_traits>

#include "hybrid.h"
#include "hybrid_mma.cuh"

namespace mb {
namespace {

using namespace hy;

__device__ __forceinline__ float log_sigmoid(float z) { return -softplus_f(-z); }

// ------------------------------------------------------------------------------------------------ decays of all rows
// Block: GC channels of a stretch of up to 128 rows, which GG groups of threads share. SUM: a stretch is a chunk, out = running sum of
// log2 a over it; else out = a - 1. RK > 0: the channel's weights sit in registers (rank <= RK).
constexpr int GC = 64, GG = 8, GROWS = HY_CHUNK / GG;

// log2 a = log2(sigmoid(z)) / tau. softplus(-z) = max(-z, 0) + log1p(exp(-|z|)); below 1/16 the logarithm comes from its series (an
// approximate one loses its digits near 1, and slow decays are made of them).
__device__ __forceinline__ float log2_sigmoid(float z) {
  const float e = ex2(-fabsf(z) * LOG2E);
  float l;
  if (e < 0.0625f) l = e * (1.f - e * (0.5f - e * (1.f / 3.f - e * (0.25f - e * (0.2f - e * (1.f / 6.f)))))) * LOG2E;
  else l = __log2f(1.f + e);
  return -(fmaxf(-z, 0.f) * LOG2E + l);
}

template <typename T, int RK, bool SUM>
__global__ void __launch_bounds__(GG * GC) gate_kernel(const HyLinear a, const int4* __restrict__ chunks, int n_rows, float* __restrict__ out, bool vec) {
  extern __shared__ __align__(16) float us[];  // [128][rank]
  __shared__ float ends[GG][GC];
  const int lane_c = threadIdx.x & (GC - 1), group = threadIdx.x / GC, ch = a.heads * a.N, c = blockIdx.y * GC + lane_c, rank = a.rank;
  const bool live = c < ch;
  int row0, n;
  if constexpr (SUM) {
    const int4 ck = chunks[blockIdx.x];
    row0 = ck.y;
    n = ck.z;
  } else {
    row0 = blockIdx.x * HY_CHUNK;
    n = min(HY_CHUNK, n_rows - row0);
  }
  const int ldu = RK > 0 ? RK : rank;
  const T* w = static_cast<const T*>(a.a2) + static_cast<long long>(live ? c : 0) * rank;
  __align__(8) float wr[RK > 0 ? RK : 2];
  constexpr int V = Vec<T>::N;
  if (RK > 0 && vec) {  // (rank a multiple of V, 16-byte aligned rows)
    if constexpr (RK > 0) {
#pragma unroll
      for (int r = 0; r < RK; r += V) {
        float x[V];
#pragma unroll
        for (int j = 0; j < V; ++j) x[j] = 0.f;
        if (r < rank) Vec<T>::load(w + r, x);
#pragma unroll
        for (int j = 0; j < V; ++j) wr[r + j] = x[j];
      }
      for (int i = threadIdx.x; i < n * (RK / V); i += GG * GC) {
        const int t = i / (RK / V), r = (i - t * (RK / V)) * V;
        float x[V];
#pragma unroll
        for (int j = 0; j < V; ++j) x[j] = 0.f;
        if (r < rank) Vec<T>::load(static_cast<const T*>(a.proj) + (row0 + t) * a.ld + a.u + r, x);
#pragma unroll
        for (int j = 0; j < V; j += 4) *reinterpret_cast<float4*>(us + t * RK + r + j) = make_float4(x[j], x[j + 1], x[j + 2], x[j + 3]);
      }
    }
  } else {
    if constexpr (RK > 0) {
#pragma unroll
      for (int r = 0; r < RK; ++r) wr[r] = r < rank ? to_f(w[r]) : 0.f;
    }
    for (int i = threadIdx.x; i < n * ldu; i += GG * GC) {
      const int t = i / ldu, r = i - t * ldu;
      us[i] = r < rank ? to_f(static_cast<const T*>(a.proj)[(row0 + t) * a.ld + a.u + r]) : 0.f;
    }
  }
  const float bias = live ? to_f(static_cast<const T*>(a.a2_bias)[c]) : 0.f;
  __syncthreads();
  const int t0 = group * GROWS, m = min(GROWS, n - t0);
  auto z_of = [&](int t) {
    if constexpr (RK > 0) {  // two products an instruction
      float2 z = make_float2(bias, 0.f);
#pragma unroll
      for (int r = 0; r < RK; r += 4) {
        const float4 u = *reinterpret_cast<const float4*>(us + t * RK + r);
        z = __ffma2_rn(make_float2(wr[r], wr[r + 1]), make_float2(u.x, u.y), z);
        z = __ffma2_rn(make_float2(wr[r + 2], wr[r + 3]), make_float2(u.z, u.w), z);
      }
      return z.x + z.y;
    } else {
      float z = bias;
      for (int r = 0; r < rank; ++r) z += to_f(w[r]) * us[t * rank + r];
      return z;
    }
  };
  float* dst = out + static_cast<long long>(row0 + t0) * ch + c;
  if constexpr (SUM) {
    float run = 0.f, v[GROWS];
#pragma unroll
    for (int t = 0; t < GROWS; ++t) {
      if (t < m) run += log2_sigmoid(z_of(t0 + t)) * a.inv_tau;
      v[t] = run;
    }
    ends[group][lane_c] = run;
    __syncthreads();
    float base = 0.f;
    for (int g = 0; g < group; ++g) base += ends[g][lane_c];
    if (!live) return;
#pragma unroll
    for (int t = 0; t < GROWS; ++t)
      if (t < m) dst[static_cast<long long>(t) * ch] = base + v[t];
  } else {
    if (!live) return;
    for (int t = 0; t < m; ++t) dst[static_cast<long long>(t) * ch] = expm1f(log_sigmoid(z_of(t0 + t)) * a.inv_tau);
  }
}

// ------------------------------------------------------------------------------------------------ sequential scan
// One warp per state row p: lane l holds columns l, l + 32, ...
template <typename T, int NR>
__global__ void __launch_bounds__(256) lin_scan_kernel(const HyLinear a, const float* __restrict__ gate, T* __restrict__ y) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int p = blockIdx.x * 8 + warp, h = blockIdx.y, seq = blockIdx.z, N = a.N;
  if (p >= a.P) return;
  const int first = a.cu[seq], n = a.cu[seq + 1] - first;
  const long long slot = state_row(a.slots, a.sequences, seq, a.status);
  float* st = a.state + (((slot < 0 ? 0 : slot) * a.heads + h) * a.P + p) * N;
  float S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) S[i] = (slot >= 0 && a.ctx[seq] > 0 && lane + 32 * i < N) ? st[lane + 32 * i] : 0.f;
  const float fixed = a.rank > 0 ? 0.f : a.decay_m1[h];
  const T* rows = static_cast<const T*>(a.proj);
  for (int t = 0; t < n; ++t) {
    const long long r = first + t;
    const T *k = rows + r * a.ld + a.k + h * N, *q = rows + r * a.ld + a.q + h * N;
    const float* e = a.rank > 0 ? gate + (r * a.heads + h) * N : nullptr;
    const float v = to_f(rows[r * a.ld + a.v + h * a.P + p]);
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int c = lane + 32 * i;
      if (c < N) {
        S[i] = fmaf(e ? e[c] : fixed, S[i], S[i]) + to_f(k[c]) * v;
        o += S[i] * to_f(q[c]);
      }
    }
    o = warp_sum(o) * a.q_scale;
    if (lane == 0) y[(r * a.heads + h) * a.P + p] = from_f<T>(o);
  }
  if (slot < 0) return;
#pragma unroll
  for (int i = 0; i < NR; ++i)
    if (lane + 32 * i < N) st[lane + 32 * i] = S[i];
}

// ------------------------------------------------------------------------------------------------ output norm and gate
// A warp per (row, head). V4: four values per access.
template <typename T>
__device__ __forceinline__ float4 load4(const T* p) {
  if constexpr (sizeof(T) == 2) {
    const uint2 q = *reinterpret_cast<const uint2*>(p);
    const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x)), y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
    return make_float4(x.x, x.y, y.x, y.y);
  } else {
    return *reinterpret_cast<const float4*>(p);
  }
}
template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v) {
  if constexpr (sizeof(T) == 2) {
    const __nv_bfloat162 x = __floats2bfloat162_rn(v.x, v.y), y = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&x), *reinterpret_cast<const uint32_t*>(&y));
  } else {
    *reinterpret_cast<float4*>(p) = v;
  }
}

template <typename T, bool V4>
__global__ void __launch_bounds__(256) lin_tail_kernel(const HyLinear a, const T* __restrict__ y, T* __restrict__ out, int ldc, unsigned units) {
  const unsigned unit = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (unit >= units) return;
  const int lane = threadIdx.x & 31, P = a.P;
  const unsigned row = unit / static_cast<unsigned>(a.heads);
  const int h = static_cast<int>(unit - row * a.heads);
  const long long t = row;
  const T* src = y + static_cast<long long>(unit) * P;
  const T* g = static_cast<const T*>(a.proj) + t * a.ld + a.g + h * P;
  const T* w = static_cast<const T*>(a.norm);
  T* dst = out + t * ldc + h * P;
  float s = 0.f;
  if constexpr (V4) {
    float4 v0 = make_float4(0.f, 0.f, 0.f, 0.f);
    if (lane * 4 < P) v0 = load4(src + lane * 4);
    float4 z0 = make_float4(0.f, 0.f, 0.f, 0.f), w0 = make_float4(1.f, 1.f, 1.f, 1.f);  // (of the first 128 columns, fetched before the sum)
    if (lane * 4 < P) {
      z0 = load4(g + lane * 4);
      if (w) w0 = load4(w + lane * 4);
    }
    s = v0.x * v0.x + v0.y * v0.y + v0.z * v0.z + v0.w * v0.w;
    for (int i = 128 + lane * 4; i < P; i += 128) {
      const float4 v = load4(src + i);
      s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    const float r = sizeof(T) == 2 ? rsqrtf(warp_sum(s) / static_cast<float>(P) + a.eps) : 1.f / sqrtf(warp_sum(s) / static_cast<float>(P) + a.eps);
    for (int i = lane * 4; i < P; i += 128) {
      float4 v = i < 128 ? v0 : load4(src + i);
      const float4 z = i < 128 ? z0 : load4(g + i), q = i < 128 ? w0 : (w ? load4(w + i) : make_float4(1.f, 1.f, 1.f, 1.f));
      v.x *= r * q.x * silu_t<T>(z.x);
      v.y *= r * q.y * silu_t<T>(z.y);
      v.z *= r * q.z * silu_t<T>(z.z);
      v.w *= r * q.w * silu_t<T>(z.w);
      store4(dst + i, v);
    }
  } else {
    for (int i = lane; i < P; i += 32) s += to_f(src[i]) * to_f(src[i]);
    const float r = 1.f / sqrtf(warp_sum(s) / static_cast<float>(P) + a.eps);
    for (int i = lane; i < P; i += 32) dst[i] = from_f<T>(to_f(src[i]) * r * (w ? to_f(w[i]) : 1.f) * silu_f(to_f(g[i])));
  }
  if (h == a.heads - 1)
    for (int i = a.heads * P + lane; i < ldc; i += 32) out[t * ldc + i] = from_f<T>(0.f);
}

// ------------------------------------------------------------------------------------------------ one token
// CTA = (head, sequence). Queries, keys and decays of the head, then the state update, then the head's output norm and gate. LPR > 0: LPR
// lanes own a state row, four columns each (N <= 4 LPR, a multiple of 4); the first U rows of every lane group are fetched before
// anything else. LPR = 0: any N.
template <typename T, int LPR>
__global__ void __launch_bounds__(LPR > 0 ? 512 : 256, 2) lin_step_kernel(const HyLinear a, const int* __restrict__ positions, T* __restrict__ out, int ldc) {
  extern __shared__ __align__(16) float sm[];
  const int h = blockIdx.x, b = blockIdx.y, P = a.P, N = a.N, Np = (N + 3) & ~3;
  float *q = sm, *k = q + Np, *e = k + Np, *o = e + Np, *u = o + ((P + 3) & ~3);  // u [rank]
  const int pos = positions[b];
  const long long slot = state_row(a.slots, a.sequences, b, threadIdx.x == 0 ? a.status : nullptr);
  if (slot < 0) return;
  const T* pr = static_cast<const T*>(a.proj) + static_cast<long long>(b) * a.ld;
  const T *qr = pr + a.q + h * N, *kr = pr + a.k + h * N, *vr = pr + a.v + h * P;
  float* st = a.state + (slot * a.heads + h) * static_cast<long long>(P) * N;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const bool fresh = pos <= 0;
  const int half = a.rot / 2;
  constexpr int U = 8;
  constexpr int RPW = LPR > 0 ? 32 / LPR : 1;  // rows a warp works on at once
  const int sub = lane & (LPR > 0 ? LPR - 1 : 0), c = sub * 4, row_of = warp * RPW + (LPR > 0 ? lane / LPR : 0), rows = nw * RPW;
  const bool own = c < N;
  float4 s[LPR > 0 ? U : 1];
  float v[LPR > 0 ? U : 1];
  auto fetch = [&](int p0) {
#pragma unroll
    for (int j = 0; j < U; ++j) {
      const int p = p0 + j * rows;
      s[LPR > 0 ? j : 0] = own && !fresh && p < P ? *reinterpret_cast<const float4*>(st + static_cast<long long>(p) * N + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      v[LPR > 0 ? j : 0] = p < P ? to_f(vr[p]) : 0.f;
    }
  };
  if constexpr (LPR > 0) fetch(row_of);
  // gate and norm weight of this thread's (first) value, needed last
  const T *g = pr + a.g + h * P, *wn = static_cast<const T*>(a.norm);
  float gv = 0.f, wv = 1.f;
  if (static_cast<int>(threadIdx.x) < P) {
    gv = to_f(g[threadIdx.x]);
    if (wn) wv = to_f(wn[threadIdx.x]);
  }
  for (int i = threadIdx.x; i < a.rank; i += blockDim.x) u[i] = to_f(pr[a.u + i]);
  // (what the chunked and sequential forms read back from rotated rows is rounded there; here it is rounded the same way)
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn, cs;
    sincosf(static_cast<float>(pos) * a.freq[i], &sn, &cs);
    const float q0 = to_f(qr[i]), q1 = to_f(qr[half + i]), k0 = to_f(kr[i]), k1 = to_f(kr[half + i]);
    q[i] = to_f(from_f<T>(q0 * cs - q1 * sn));
    q[half + i] = to_f(from_f<T>(q1 * cs + q0 * sn));
    k[i] = to_f(from_f<T>((k0 * cs - k1 * sn) * a.k_scale));
    k[half + i] = to_f(from_f<T>((k1 * cs + k0 * sn) * a.k_scale));
  }
  for (int i = 2 * half + threadIdx.x; i < N; i += blockDim.x) {
    q[i] = to_f(qr[i]);
    k[i] = a.k_scale == 1.f ? to_f(kr[i]) : to_f(from_f<T>(to_f(kr[i]) * a.k_scale));
  }
  if (a.rank > 0) {
    constexpr int V = Vec<T>::N;
    const bool vec = a.rank % V == 0;
    for (int i0 = 0; i0 < N; i0 += blockDim.x) {
      const int i = i0 + threadIdx.x, ch = h * N + min(i, N - 1);
      const T* w = static_cast<const T*>(a.a2) + static_cast<long long>(ch) * a.rank;
      float z = to_f(static_cast<const T*>(a.a2_bias)[ch]), x[V];
      if (vec) Vec<T>::load(w, x);  // (in flight over the barrier)
      if (i0 == 0) __syncthreads();
      if (i >= N) continue;
      int r = 0;
      if (vec)
        for (; r < a.rank; r += V) {
          if (r > 0) Vec<T>::load(w + r, x);
#pragma unroll
          for (int j = 0; j < V; ++j) z += x[j] * u[r + j];
        }
      for (; r < a.rank; ++r) z += to_f(w[r]) * u[r];
      e[i] = expm1f(log_sigmoid(z) * a.inv_tau);
    }
  } else {
    for (int i = threadIdx.x; i < N; i += blockDim.x) e[i] = a.decay_m1[h];
  }
  __syncthreads();
  if constexpr (LPR > 0) {
    float4 kv = make_float4(0.f, 0.f, 0.f, 0.f), qv = kv, ev = kv;
    if (own) {
      kv = *reinterpret_cast<const float4*>(k + c);
      qv = *reinterpret_cast<const float4*>(q + c);
      ev = *reinterpret_cast<const float4*>(e + c);
    }
    for (int p0 = row_of; p0 - row_of < P; p0 += U * rows) {
      if (p0 != row_of) fetch(p0);
      float acc[U];
#pragma unroll
      for (int j = 0; j < U; ++j) {
        s[j].x = fmaf(ev.x, s[j].x, s[j].x) + kv.x * v[j];
        s[j].y = fmaf(ev.y, s[j].y, s[j].y) + kv.y * v[j];
        s[j].z = fmaf(ev.z, s[j].z, s[j].z) + kv.z * v[j];
        s[j].w = fmaf(ev.w, s[j].w, s[j].w) + kv.w * v[j];
        acc[j] = s[j].x * qv.x + s[j].y * qv.y + s[j].z * qv.z + s[j].w * qv.w;
        if (own && p0 + j * rows < P) *reinterpret_cast<float4*>(st + static_cast<long long>(p0 + j * rows) * N + c) = s[j];
      }
#pragma unroll
      for (int j = 0; j < U; ++j) {
#pragma unroll
        for (int off = LPR / 2; off > 0; off >>= 1) acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], off);
        if (sub == 0 && p0 + j * rows < P) o[p0 + j * rows] = acc[j] * a.q_scale;
      }
    }
  } else {
    for (int p = warp; p < P; p += nw) {
      float acc = 0.f;
      const float vp = to_f(vr[p]);
      float* row = st + static_cast<long long>(p) * N;
      for (int i = lane; i < N; i += 32) {
        const float s0 = fresh ? 0.f : row[i];
        const float s1 = fmaf(e[i], s0, s0) + k[i] * vp;
        row[i] = s1;
        acc += s1 * q[i];
      }
      acc = warp_sum(acc);
      if (lane == 0) o[p] = acc * a.q_scale;
    }
  }
  __syncthreads();
  float ss = 0.f;  // (every warp adds up all of the head)
  for (int p = lane; p < P; p += 32) ss += o[p] * o[p];
  const float r = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(P) + a.eps);
  T* dst = out + static_cast<long long>(b) * ldc;
  for (int p = threadIdx.x; p < P; p += blockDim.x) {
    if (p >= static_cast<int>(blockDim.x)) {
      gv = to_f(g[p]);
      if (wn) wv = to_f(wn[p]);
    }
    dst[h * P + p] = from_f<T>(o[p] * r * wv * silu_f(gv));
  }
  if (h == a.heads - 1)
    for (int i = a.heads * P + threadIdx.x; i < ldc; i += blockDim.x) dst[i] = from_f<T>(0.f);
}

// ------------------------------------------------------------------------------------------------ chunks (bf16)
constexpr int Q = HY_CHUNK;
constexpr int CW = 8;          // warps of the state kernel
constexpr int OW = 16;         // warps of the output kernel
constexpr int PAD = 8;
constexpr int NMAX = 128;      // key channels
constexpr int PBLK = 128;      // value columns per CTA
constexpr float SPAN = 60.f;   // log2 units a channel may move from the chunk's reference

// bf16 x 8 from global memory, with a running-sum row beside it; columns past N and rows past n give zeros
struct Eight {
  float v[8], c[8];
};
template <bool VEC>
__device__ __forceinline__ Eight load8(const bf16* __restrict__ src, const float* __restrict__ sums, int col, int N, bool row) {
  Eight x;
#pragma unroll
  for (int j = 0; j < 8; ++j) x.v[j] = x.c[j] = 0.f;
  if (!row || col >= N) return x;
  if constexpr (VEC) {
    Vec<bf16>::load(src + col, x.v);
    const float4 a = *reinterpret_cast<const float4*>(sums + col), b = *reinterpret_cast<const float4*>(sums + col + 4);
    x.c[0] = a.x; x.c[1] = a.y; x.c[2] = a.z; x.c[3] = a.w;
    x.c[4] = b.x; x.c[5] = b.y; x.c[6] = b.z; x.c[7] = b.w;
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (col + j < N) {
        x.v[j] = to_f(src[col + j]);
        x.c[j] = sums[col + j];
      }
  }
  return x;
}
__device__ __forceinline__ void put8(const float (&v)[8], bf16* hi, bf16* lo) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) split2(v[2 * j], v[2 * j + 1], h[j], l[j]);
  *reinterpret_cast<uint4*>(hi) = make_uint4(h[0], h[1], h[2], h[3]);
  *reinterpret_cast<uint4*>(lo) = make_uint4(l[0], l[1], l[2], l[3]);
}

// (1) work[chunk, h, p, c] = sum_t v_t[p] k_t[c] 2^(sum_end - sum_t);  decay[chunk, h] = {2^sum_end, 2^reference (1 in a wide chunk)}
template <int PT, bool VEC>
__global__ void __launch_bounds__(CW * 32, 2) lin_state_kernel(const HyLinear a, const float* __restrict__ gate, const int4* __restrict__ chunks,
                                                               float* __restrict__ work, float* __restrict__ decay, int* __restrict__ wide,
                                                               bool vec_v) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int4 ck = chunks[blockIdx.x];
  const int row0 = ck.y, n = ck.z, h = blockIdx.y, P = a.P, N = a.N, NP = (N + 15) / 16 * 16, p_base = blockIdx.z * PBLK;
  const int ch = a.heads * N, pw = min(P - p_base, PBLK);
  constexpr int PP = PT * 16, ldv = PP + PAD;
  const int ldk = NP + PAD;
  bf16* Vs = reinterpret_cast<bf16*>(raw);   // [Q][ldv]
  bf16* Kh = Vs + Q * ldv;                   // [Q][ldk] weighted keys, high part
  bf16* Kl = Kh + Q * ldk;
  __shared__ float ends[NMAX];
  const bf16* rows = static_cast<const bf16*>(a.proj) + row0 * a.ld;
  const float* sums = gate + static_cast<long long>(row0) * ch + h * N;
  load_tile<CW * 32>(rows + a.v + h * P + p_base, a.ld, n, pw, Q, PP, Vs, ldv, vec_v);
  bool far = false;
  if (static_cast<int>(threadIdx.x) < NMAX) {
    const int c = threadIdx.x;
    float end = 0.f, mid = 0.f;
    if (c < N) {
      end = sums[static_cast<long long>(n - 1) * ch + c];
      mid = sums[static_cast<long long>(min(n - 1, Q / 2 - 1)) * ch + c];
    }
    ends[c] = end;
    far = !(-mid <= SPAN && mid - end <= SPAN);
  }
  const bool w = __syncthreads_or(far) != 0;
  const long long at = static_cast<long long>(blockIdx.x) * a.heads + h;
  if (p_base == 0) {
    for (int c = threadIdx.x; c < N; c += CW * 32) {
      decay[at * 2 * N + c] = ex2(ends[c]);
      decay[(at * 2 + 1) * N + c] = w ? 1.f : ex2(sums[static_cast<long long>(min(n - 1, Q / 2 - 1)) * ch + c]);
    }
    if (threadIdx.x == 0) wide[at] = w ? 1 : 0;
  }
  const int per = NP / 8;
  for (int i = threadIdx.x; i < Q * per; i += CW * 32) {
    const int t = i / per, c = (i - t * per) * 8;
    Eight x = load8<VEC>(rows + t * a.ld + a.k + h * N, sums + static_cast<long long>(t) * ch, c, N, t < n);
#pragma unroll
    for (int j = 0; j < 8; ++j) x.v[j] *= ex2(ends[c + j] - x.c[j]);
    put8(x.v, Kh + t * ldk + c, Kl + t * ldk + c);
  }
  cp_wait_all();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nt = (NP + 63) / 64;
  float* out = work + at * P * N + static_cast<long long>(p_base) * N;
  for (int unit = warp; unit < PT * nt; unit += CW) {
    const int m0 = (unit % PT) * 16, n0 = (unit / PT) * 64;
    if (m0 >= pw) continue;
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll 2
    for (int k0 = 0; k0 < n; k0 += 16) {
      uint32_t av[4];
      const int ar = k0 + (lane & 7) + ((lane >> 4) << 3), ac = m0 + (((lane >> 3) & 1) << 3);
      ldsm4t(s_u32(Vs + ar * ldv + ac), av);
#pragma unroll
      for (int jp = 0; jp < 4; ++jp) {
        if (n0 + jp * 16 >= NP) break;
        uint32_t b[4], d[4];
        const int br = k0 + (lane & 7) + (((lane >> 3) & 1) << 3), bc = n0 + jp * 16 + ((lane >> 4) << 3);
        ldsm4t(s_u32(Kh + br * ldk + bc), b);
        ldsm4t(s_u32(Kl + br * ldk + bc), d);
        mma(acc[2 * jp], av, b[0], b[1]);
        mma(acc[2 * jp], av, d[0], d[1]);
        mma(acc[2 * jp + 1], av, b[2], b[3]);
        mma(acc[2 * jp + 1], av, d[2], d[3]);
      }
    }
    const int p0 = m0 + (lane >> 2);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int c = n0 + j * 8 + (lane & 3) * 2;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int p = p0 + i * 8;
        if (p >= pw) continue;
        float* dst = out + static_cast<long long>(p) * N + c;
        if ((N & 1) == 0) {
          if (c < N) *reinterpret_cast<float2*>(dst) = make_float2(acc[j][2 * i], acc[j][2 * i + 1]);
        } else {
          if (c < N) dst[0] = acc[j][2 * i];
          if (c + 1 < N) dst[1] = acc[j][2 * i + 1];
        }
      }
    }
  }
}

// (3) outputs of a chunk (the scan over chunks (2) is Mamba-2's). The lower triangle has 36 blocks of 16 x 16 tokens, whose weights are
// kept as A fragments (two bf16 terms); a warp then takes the row tiles (w, 7 - w), nine blocks, and 16 * PH value columns.
template <int PH, bool VEC>
__global__ void __launch_bounds__(OW * 32, 1) lin_out_kernel(const HyLinear a, const float* __restrict__ gate, const int4* __restrict__ chunks,
                                                             const int* __restrict__ wide, const bf16* __restrict__ before,
                                                             bf16* __restrict__ y, bool vec_v, bool vec_s) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int4 ck = chunks[blockIdx.x];
  const int seq = ck.x, row0 = ck.y, n = ck.z, h = blockIdx.y, P = a.P, N = a.N, NP = (N + 15) / 16 * 16, p_base = blockIdx.z * PBLK;
  const int ch = a.heads * N, pw = min(P - p_base, PBLK);
  constexpr int PP = PH * 64, ldv = PP + PAD;
  const int ldk = NP + PAD;
  uint4* Gs = reinterpret_cast<uint4*>(raw);             // [36][2][32 lanes]
  bf16* Qh = reinterpret_cast<bf16*>(Gs + 36 * 64);      // [Q][ldk]
  bf16* Ql = Qh + Q * ldk;
  bf16* Kh = Ql + Q * ldk;                               // [Q][ldk]; the carried state [PP][ldk] after the weights are done
  bf16* Kl = Kh + Q * ldk;
  bf16* Vs = Kl + Q * ldk;                               // [Q][ldv]
  const bool carried = ck.w > 0 || a.ctx[seq] > 0;
  const long long at = static_cast<long long>(blockIdx.x) * a.heads + h;
  const bool w = wide[at] != 0;
  const bf16* rows = static_cast<const bf16*>(a.proj) + row0 * a.ld;
  const float* sums = gate + static_cast<long long>(row0) * ch + h * N;
  const int per = NP / 8, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  load_tile<OW * 32>(rows + a.v + h * P + p_base, a.ld, n, pw, Q, PP, Vs, ldv, vec_v);
  cp_commit();
  const int a_row = lane & 15, a_col = (lane >> 4) << 3;
  const int b_row = (lane & 7) + ((lane >> 4) << 3), b_col = ((lane >> 3) & 1) << 3;    // [n][k] operands
  const int v_row = (lane & 7) + (((lane >> 3) & 1) << 3), v_col = (lane >> 4) << 3;    // [k][n] operands

  // queries (or keys: sign -1) times 2^(sum - reference): the reference is row `ref` of the sums, none for ref < 0
  auto weigh = [&](int col0, int rows_n, int ref, int ref_step, float sign, float scale, bf16* hi, bf16* lo) {
    for (int i = threadIdx.x; i < rows_n * per; i += OW * 32) {
      const int t = i / per, c = (i - t * per) * 8;
      Eight x = load8<VEC>(rows + t * a.ld + col0, sums + static_cast<long long>(t) * ch, c, N, t < n);
      const int rr = ref_step > 0 ? t / ref_step * ref_step - 1 : ref;
      Eight r;
#pragma unroll
      for (int j = 0; j < 8; ++j) r.c[j] = 0.f;
      if (rr >= 0) r = load8<VEC>(rows, sums + static_cast<long long>(rr) * ch, c, N, t < n);
#pragma unroll
      for (int j = 0; j < 8; ++j) x.v[j] *= scale * ex2(sign * (x.c[j] - r.c[j]));
      put8(x.v, hi + t * ldk + c, lo + t * ldk + c);
    }
  };
  // weights of block (r, s) from the two factors
  auto scores = [&](int r, int s, float (&g0)[4], float (&g1)[4]) {
#pragma unroll
    for (int j = 0; j < 4; ++j) g0[j] = g1[j] = 0.f;
    const int qo = (r * 16 + a_row) * ldk + a_col, ko = (s * 16 + b_row) * ldk + b_col;
#pragma unroll 2
    for (int k0 = 0; k0 < NP; k0 += 16) {
      uint32_t qh[4], ql[4], kh[4], kl[4];
      ldsm4(s_u32(Qh + qo + k0), qh);
      ldsm4(s_u32(Ql + qo + k0), ql);
      ldsm4(s_u32(Kh + ko + k0), kh);
      ldsm4(s_u32(Kl + ko + k0), kl);
      mma(g0, qh, kh[0], kh[1]);
      mma(g1, qh, kh[2], kh[3]);
      mma(g0, qh, kl[0], kl[1]);
      mma(g1, qh, kl[2], kl[3]);
      mma(g0, ql, kh[0], kh[1]);
      mma(g1, ql, kh[2], kh[3]);
    }
  };
  // to A fragments; accumulator layout = A-operand layout
  auto keep = [&](int r, int s, const float (&g0)[4], const float (&g1)[4]) {
    const int blk = r * (r + 1) / 2 + s;
    float v[8] = {g0[0], g0[1], g0[2], g0[3], g1[0], g1[1], g1[2], g1[3]};
    if (r == s) {  // only tokens up to t
      const int t = lane >> 2, c = (lane & 3) * 2;
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (c + (j >> 2) * 8 + (j & 1) > t + ((j >> 1) & 1) * 8) v[j] = 0.f;
    }
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) split2(v[2 * j], v[2 * j + 1], hi[j], lo[j]);
    Gs[blk * 64 + lane] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    Gs[blk * 64 + 32 + lane] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  };

  if (!w) {
    const int ref = min(n - 1, Q / 2 - 1);
    weigh(a.q + h * N, Q, ref, 0, 1.f, a.q_scale, Qh, Ql);
    weigh(a.k + h * N, Q, ref, 0, -1.f, 1.f, Kh, Kl);
    __syncthreads();
    for (int blk = warp; blk < 36; blk += OW) {
      int r = 0;
      while ((r + 1) * (r + 2) / 2 <= blk) ++r;
      const int s = blk - r * (r + 1) / 2;
      float g0[4], g1[4];
      scores(r, s, g0, g1);
      keep(r, s, g0, g1);
    }
    __syncthreads();
  } else {
    weigh(a.q + h * N, Q, 0, 16, 1.f, a.q_scale, Qh, Ql);  // from the end of the 16 tokens before
    for (int r = 1; r * 16 < n; ++r) {
      __syncthreads();  // the keys of the row tile before have been read
      weigh(a.k + h * N, r * 16, r * 16 - 1, 0, -1.f, 1.f, Kh, Kl);
      __syncthreads();
      for (int s = warp; s < r; s += OW) {
        float g0[4], g1[4];
        scores(r, s, g0, g1);
        keep(r, s, g0, g1);
      }
    }
    if (warp < 8 && warp * 16 < n) {  // blocks on the diagonal: every product on its own
      const int t0 = warp * 16 + (lane >> 2), s0 = warp * 16 + (lane & 3) * 2;
      float g[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) g[j] = 0.f;
      for (int c = 0; c < N; ++c) {
        float qv[2], qc[2], kv[4], kc[4];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int t = min(t0 + i * 8, n - 1);
          qv[i] = to_f(rows[t * a.ld + a.q + h * N + c]);
          qc[i] = sums[static_cast<long long>(t) * ch + c];
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int s = min(s0 + (i >> 1) * 8 + (i & 1), n - 1);
          kv[i] = to_f(rows[s * a.ld + a.k + h * N + c]);
          kc[i] = sums[static_cast<long long>(s) * ch + c];
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const int i = (j >> 1) & 1, k = (j >> 2) * 2 + (j & 1);
          g[j] += qv[i] * kv[k] * ex2(fminf(qc[i] - kc[k], 0.f));  // (positive only above the diagonal, which is dropped)
        }
      }
      const float g0[4] = {g[0] * a.q_scale, g[1] * a.q_scale, g[2] * a.q_scale, g[3] * a.q_scale};
      const float g1[4] = {g[4] * a.q_scale, g[5] * a.q_scale, g[6] * a.q_scale, g[7] * a.q_scale};
      keep(warp, warp, g0, g1);
    }
    __syncthreads();
    weigh(a.q + h * N, Q, -1, 0, 1.f, a.q_scale, Qh, Ql);  // from the chunk's start: what meets the carried state
    __syncthreads();
  }
  if (carried) {
    const bf16* src = before + at * 2 * P * N + static_cast<long long>(p_base) * N;
    load_tile<OW * 32>(src, N, pw, N, PP, NP, Kh, ldk, vec_s);
    load_tile<OW * 32>(src + static_cast<long long>(P) * N, N, pw, N, PP, NP, Kl, ldk, vec_s);
  }
  cp_wait_all();
  __syncthreads();
  const int pg = warp >> 2, ta = warp & 3, tb = 7 - ta;     // column group, row tiles
  const int pc0 = pg * PH * 16;                              // first column of this warp
  if (pc0 >= pw) return;
#pragma unroll 1
  for (int half = 0; half < 2; ++half) {
    const int tile = half == 0 ? ta : tb;
    if (tile * 16 >= n) continue;
    float o[2 * PH][4];
#pragma unroll
    for (int j = 0; j < 2 * PH; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    if (carried) {
      const int qo = (tile * 16 + a_row) * ldk + a_col, so = (pc0 + b_row) * ldk + b_col;
#pragma unroll 2
      for (int k0 = 0; k0 < NP; k0 += 16) {
        uint32_t qh[4], ql[4];
        ldsm4(s_u32(Qh + qo + k0), qh);
        ldsm4(s_u32(Ql + qo + k0), ql);
#pragma unroll
        for (int jp = 0; jp < PH; ++jp) {
          uint32_t b[4], c[4];
          ldsm4(s_u32(Kh + so + jp * 16 * ldk + k0), b);
          ldsm4(s_u32(Kl + so + jp * 16 * ldk + k0), c);
          mma(o[2 * jp], qh, b[0], b[1]);
          mma(o[2 * jp + 1], qh, b[2], b[3]);
          mma(o[2 * jp], qh, c[0], c[1]);
          mma(o[2 * jp + 1], qh, c[2], c[3]);
          mma(o[2 * jp], ql, b[0], b[1]);
          mma(o[2 * jp + 1], ql, b[2], b[3]);
        }
      }
    }
    const uint4* gp = Gs + tile * (tile + 1) / 2 * 64 + lane;
#pragma unroll 2
    for (int st = 0; st <= tile; ++st) {
      const uint4 h4 = gp[st * 64], l4 = gp[st * 64 + 32];
      const uint32_t wh[4] = {h4.x, h4.y, h4.z, h4.w}, wl[4] = {l4.x, l4.y, l4.z, l4.w};
      const uint32_t va = s_u32(Vs + (st * 16 + v_row) * ldv + pc0 + v_col);
#pragma unroll
      for (int jp = 0; jp < PH; ++jp) {
        uint32_t b[4];
        ldsm4t(va + jp * 32, b);
        mma(o[2 * jp], wh, b[0], b[1]);
        mma(o[2 * jp + 1], wh, b[2], b[3]);
        mma(o[2 * jp], wl, b[0], b[1]);
        mma(o[2 * jp + 1], wl, b[2], b[3]);
      }
    }
    const int r0 = tile * 16 + (lane >> 2);
#pragma unroll
    for (int j = 0; j < 2 * PH; ++j) {
      const int p = pc0 + j * 8 + (lane & 3) * 2;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = r0 + i * 8;
        if (t >= n) continue;
        bf16* dst = y + (static_cast<long long>(row0 + t) * a.heads + h) * P + p_base + p;
        if ((P & 1) == 0) {
          if (p < pw) *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(o[j][2 * i], o[j][2 * i + 1]);
        } else {
          if (p < pw) dst[0] = __float2bfloat16(o[j][2 * i]);
          if (p + 1 < pw) dst[1] = __float2bfloat16(o[j][2 * i + 1]);
        }
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ launches
template <typename T, int RK, bool SUM>
int gate_rk(const HyLinear& a, const int* chunks, int n_chunks, int rows, float* out, cudaStream_t s) {
  const size_t smem = sizeof(float) * HY_CHUNK * static_cast<size_t>(RK > 0 ? RK : a.rank);
  auto kern = gate_kernel<T, RK, SUM>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  const unsigned x = SUM ? n_chunks : (rows + HY_CHUNK - 1) / HY_CHUNK;
  const bool vec = a.rank % Vec<T>::N == 0 && a.u % Vec<T>::N == 0 && aligned16<T>(a.proj, a.ld) && aligned16<T>(a.a2, a.rank);
  kern<<<dim3(x, (a.heads * a.N + GC - 1) / GC), GG * GC, smem, s>>>(a, reinterpret_cast<const int4*>(chunks), rows, out, vec);
  return static_cast<int>(cudaGetLastError());
}
template <typename T, bool SUM>
int gate_t(const HyLinear& a, const int* chunks, int n_chunks, int rows, float* out, cudaStream_t s) {
  if (a.rank <= 16) return gate_rk<T, 16, SUM>(a, chunks, n_chunks, rows, out, s);
  if (a.rank <= 32) return gate_rk<T, 32, SUM>(a, chunks, n_chunks, rows, out, s);
  if (a.rank <= 64) return gate_rk<T, 64, SUM>(a, chunks, n_chunks, rows, out, s);
  return gate_rk<T, 0, SUM>(a, chunks, n_chunks, rows, out, s);
}

template <typename T>
int lin_scan_t(const HyLinear& a, const float* gate, void* y, cudaStream_t s) {
  const dim3 grid((a.P + 7) / 8, a.heads, a.nseq);
  T* out = static_cast<T*>(y);
  if (a.N <= 32) lin_scan_kernel<T, 1><<<grid, 256, 0, s>>>(a, gate, out);
  else if (a.N <= 64) lin_scan_kernel<T, 2><<<grid, 256, 0, s>>>(a, gate, out);
  else if (a.N <= 128) lin_scan_kernel<T, 4><<<grid, 256, 0, s>>>(a, gate, out);
  else if (a.N <= 256) lin_scan_kernel<T, 8><<<grid, 256, 0, s>>>(a, gate, out);
  else if (a.N <= 1024) lin_scan_kernel<T, 32><<<grid, 256, 0, s>>>(a, gate, out);
  else return static_cast<int>(cudaErrorInvalidValue);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int lin_tail_t(const HyLinear& a, const void* y, int rows, void* out, int ldc, cudaStream_t s) {
  const long long units = static_cast<long long>(rows) * a.heads;
  if (units == 0) return 0;
  if (units > 0x7fffffffll) return static_cast<int>(cudaErrorInvalidValue);
  const bool v4 = (a.P | a.g | ldc) % 4 == 0 && a.ld % 4 == 0;
  const unsigned blocks = static_cast<unsigned>((units + 7) / 8);
  if (v4) lin_tail_kernel<T, true><<<blocks, 256, 0, s>>>(a, static_cast<const T*>(y), static_cast<T*>(out), ldc, static_cast<unsigned>(units));
  else lin_tail_kernel<T, false><<<blocks, 256, 0, s>>>(a, static_cast<const T*>(y), static_cast<T*>(out), ldc, static_cast<unsigned>(units));
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int lin_step_t(const HyLinear& a, const int* positions, int B, void* out, int ldc, cudaStream_t s) {
  const size_t smem = sizeof(float) * (static_cast<size_t>(3) * ((a.N + 3) & ~3) + ((a.P + 3) & ~3) + a.rank);
  auto go = [&](auto kern, int lpr) -> int {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    int threads = 256;
    if (lpr > 0)  // eight rows per lane group, as far as a block reaches
      for (threads = 128; threads < 512 && threads / lpr * 8 < a.P;) threads *= 2;
    kern<<<dim3(a.heads, B), threads, smem, s>>>(a, positions, static_cast<T*>(out), ldc);
    return static_cast<int>(cudaGetLastError());
  };
  if (a.N % 4 != 0 || a.N > 128) return go(lin_step_kernel<T, 0>, 0);
  if (a.N > 64) return go(lin_step_kernel<T, 32>, 32);
  if (a.N > 32) return go(lin_step_kernel<T, 16>, 16);
  return go(lin_step_kernel<T, 8>, 8);
}

size_t state_smem(int PT, int N) { return sizeof(bf16) * Q * (static_cast<size_t>(PT) * 16 + PAD + 2 * ((N + 15) / 16 * 16 + PAD)); }
size_t out_smem(int PH, int N) {
  return 36 * 64 * sizeof(uint4) + sizeof(bf16) * Q * (4 * (static_cast<size_t>((N + 15) / 16 * 16) + PAD) + PH * 64 + PAD);
}

template <int PT, bool VEC>
int launch_state(const HyLinear& a, const float* gate, const int4* ck, int n, float* work, float* decay, int* wide, bool vec_v, cudaStream_t s) {
  const size_t smem = state_smem(PT, a.N);
  auto kern = lin_state_kernel<PT, VEC>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(n, a.heads, (a.P + PBLK - 1) / PBLK), CW * 32, smem, s>>>(a, gate, ck, work, decay, wide, vec_v);
  return static_cast<int>(cudaGetLastError());
}
template <int PH, bool VEC>
int launch_out(const HyLinear& a, const float* gate, const int4* ck, int n, const int* wide, const bf16* before, bf16* y, bool vec_v, bool vec_s,
               cudaStream_t s) {
  const size_t smem = out_smem(PH, a.N);
  auto kern = lin_out_kernel<PH, VEC>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(n, a.heads, (a.P + PBLK - 1) / PBLK), OW * 32, smem, s>>>(a, gate, ck, wide, before, y, vec_v, vec_s);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace

int hy_linear_gate(bool f32, const HyLinear& a, const int* chunks, int n_chunks, int T, float* out, cudaStream_t s) {
  if (T == 0) return 0;
  if (chunks) return f32 ? gate_t<float, true>(a, chunks, n_chunks, T, out, s) : gate_t<bf16, true>(a, chunks, n_chunks, T, out, s);
  return f32 ? gate_t<float, false>(a, chunks, 0, T, out, s) : gate_t<bf16, false>(a, chunks, 0, T, out, s);
}
int hy_linear_scan(bool f32, const HyLinear& a, const float* gate, void* y, cudaStream_t s) {
  return f32 ? lin_scan_t<float>(a, gate, y, s) : lin_scan_t<bf16>(a, gate, y, s);
}
int hy_linear_tail(bool f32, const HyLinear& a, const void* y, int T, void* out, int ldc, cudaStream_t s) {
  return f32 ? lin_tail_t<float>(a, y, T, out, ldc, s) : lin_tail_t<bf16>(a, y, T, out, ldc, s);
}
int hy_linear_step(bool f32, const HyLinear& a, const int* positions, int B, void* out, int ldc, cudaStream_t s) {
  return f32 ? lin_step_t<float>(a, positions, B, out, ldc, s) : lin_step_t<bf16>(a, positions, B, out, ldc, s);
}

bool hy_linear_chunks_supported(int P, int N) {
  return P >= 1 && N >= 1 && N <= NMAX && out_smem(P <= 64 ? 1 : 2, N) <= 227 * 1024 && state_smem(8, N) <= 227 * 1024;
}

int hy_linear_chunks(const HyLinear& a, const float* gate, const int* chunks, int n_chunks, const int* first_chunk, float* work, float* decay,
                     int* wide, void* before, void* y_, cudaStream_t s) {
  if (!hy_linear_chunks_supported(a.P, a.N)) return static_cast<int>(cudaErrorInvalidValue);
  const int4* ck = reinterpret_cast<const int4*>(chunks);
  bf16* y = static_cast<bf16*>(y_);
  const bool rows16 = aligned16<bf16>(a.proj, a.ld);
  const bool vec = rows16 && (a.N | a.k | a.q) % 8 == 0, vec_v = rows16 && (a.P | a.v) % 8 == 0, vec_s = a.N % 8 == 0;
  const int w = a.P < PBLK ? a.P : PBLK;
  int rc;
  auto state = [&](auto v) -> int {
    constexpr bool V = decltype(v)::value;
    if (w <= 32) return launch_state<2, V>(a, gate, ck, n_chunks, work, decay, wide, vec_v, s);
    if (w <= 64) return launch_state<4, V>(a, gate, ck, n_chunks, work, decay, wide, vec_v, s);
    if (w <= 96) return launch_state<6, V>(a, gate, ck, n_chunks, work, decay, wide, vec_v, s);
    return launch_state<8, V>(a, gate, ck, n_chunks, work, decay, wide, vec_v, s);
  };
  auto outs = [&](auto v) -> int {
    constexpr bool V = decltype(v)::value;
    const bf16* bf = static_cast<const bf16*>(before);
    return w <= 64 ? launch_out<1, V>(a, gate, ck, n_chunks, wide, bf, y, vec_v, vec_s, s) : launch_out<2, V>(a, gate, ck, n_chunks, wide, bf, y, vec_v, vec_s, s);
  };
  rc = vec ? state(std::true_type{}) : state(std::false_type{});
  if (rc != 0) return rc;
  HyMamba m = {};
  m.heads = a.heads; m.P = a.P; m.N = a.N; m.groups = a.heads;
  m.state = a.state; m.sequences = a.sequences;
  m.ctx = a.ctx; m.slots = a.slots; m.nseq = a.nseq; m.status = a.status;
  rc = hy_chunk_pass(m, first_chunk, decay, true, work, before, s);
  if (rc != 0) return rc;
  return vec ? outs(std::true_type{}) : outs(std::false_type{});
}

}  // namespace mb
