// Row-wise kernels of sequential blocks (a norm before and after every sublayer): head-wise rotation / norm of projected rows, the
// gated activation between the feed-forward's products, and the residual update with both norms around it.
#include "hybrid.h"
#include "hybrid_common.cuh"

namespace mb {
namespace {

using namespace hy;

// ------------------------------------------------------------------------------------------------ heads of a row
template <typename T>
struct Pair;  // two consecutive values, one load
template <>
struct Pair<float> {
  static __device__ __forceinline__ float2 load(const float* p) { return *reinterpret_cast<const float2*>(p); }
  static __device__ __forceinline__ void store(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
};
template <>
struct Pair<bf16> {
  static __device__ __forceinline__ float2 load(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
  static __device__ __forceinline__ void store(bf16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }
};

// One head by one warp. V2: two values per access (everything even).
template <typename T, typename O, bool V2>
__device__ __forceinline__ void head_row(const HyHeadOp& op, const T* __restrict__ src, O* __restrict__ dst, float pos, float eps) {
  const int lane = threadIdx.x & 31, half = op.rot / 2;
  constexpr int W = V2 ? 2 : 1;
  float scale = op.scale;
  if (op.unit) {  // (a rotation keeps the length, so that it is measured before)
    float s = 0.f;
    for (int i = lane * W; i < op.dim; i += 32 * W) {
      if constexpr (V2) {
        const float2 v = Pair<T>::load(src + i);
        s += v.x * v.x + v.y * v.y;
      } else {
        s += to_f(src[i]) * to_f(src[i]);
      }
    }
    scale /= sqrtf(warp_sum(s) / static_cast<float>(op.dim) + eps);
  }
  for (int i = lane * W; i < half; i += 32 * W) {
    float sn[W], cs[W];
#pragma unroll
    for (int k = 0; k < W; ++k) sincosf(pos * op.freq[i + k], &sn[k], &cs[k]);
    if constexpr (V2) {
      const float2 u = Pair<T>::load(src + i), v = Pair<T>::load(src + half + i);
      Pair<O>::store(dst + i, make_float2((u.x * cs[0] - v.x * sn[0]) * scale, (u.y * cs[1] - v.y * sn[1]) * scale));
      Pair<O>::store(dst + half + i, make_float2((v.x * cs[0] + u.x * sn[0]) * scale, (v.y * cs[1] + u.y * sn[1]) * scale));
    } else {
      const float u = to_f(src[i]), v = to_f(src[half + i]);
      dst[i] = from_f<O>((u * cs[0] - v * sn[0]) * scale);
      dst[half + i] = from_f<O>((v * cs[0] + u * sn[0]) * scale);
    }
  }
  for (int i = op.rot + lane * W; i < op.dim; i += 32 * W) {
    if constexpr (V2) {
      const float2 v = Pair<T>::load(src + i);
      Pair<O>::store(dst + i, make_float2(v.x * scale, v.y * scale));
    } else {
      dst[i] = from_f<O>(to_f(src[i]) * scale);
    }
  }
  for (int i = op.dim + lane; i < op.pitch; i += 32) dst[i] = from_f<O>(0.f);
}

template <typename T, bool V2>
__global__ void __launch_bounds__(256) head_rows_kernel(const HyHeadRows a, int per_row, long long units) {
  const long long unit = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (unit >= units) return;
  const int lane = threadIdx.x & 31;
  const long long t = unit / per_row;
  int h = static_cast<int>(unit - t * per_row), o = 0;
  while (h >= a.op[o].heads) h -= a.op[o++].heads;
  const HyHeadOp& op = a.op[o];
  long long row = t;
  if (op.by_slot) {
    row = a.slots[t];
    if (row < 0 || row >= a.num_slots) {
      if (lane == 0 && a.status) atomicCAS(a.status, 0, 9);
      return;
    }
  }
  const T* src = static_cast<const T*>(a.proj) + t * a.ld + op.src + h * op.dim;
  const long long at = row * op.ld + op.col + h * op.pitch;
  const float pos = op.rot > 0 ? static_cast<float>(a.positions[t]) : 0.f;
  const int extra = h == op.heads - 1 ? op.tail : 0;
  if (op.f32) {
    float* dst = static_cast<float*>(op.dst) + at;
    head_row<T, float, V2>(op, src, dst, pos, a.eps);
    for (int i = lane; i < extra; i += 32) dst[op.pitch + i] = 0.f;
  } else {
    T* dst = static_cast<T*>(op.dst) + at;
    head_row<T, T, V2>(op, src, dst, pos, a.eps);
    for (int i = lane; i < extra; i += 32) dst[op.pitch + i] = from_f<T>(0.f);
  }
}

// ------------------------------------------------------------------------------------------------ gated activation
template <typename T, int ACT>
__global__ void __launch_bounds__(256) gated_act_kernel(const T* __restrict__ proj, long long ld, int gate, int up, int ff, int ldo,
                                                        T* __restrict__ out, bool vec, long long units, int per_row) {
  constexpr int N = Vec<T>::N;
  const long long unit = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (unit >= units) return;
  const long long t = unit / per_row;
  const int c0 = static_cast<int>(unit - t * per_row) * N;
  const T* row = proj + t * ld;
  T* dst = out + t * ldo;
  auto act = [](float g, float u) { return (ACT == 1 ? fmaxf(g, 0.f) : silu_f(g)) * u; };
  if (vec && c0 + N <= ff) {
    float g[N], u[N];
    Vec<T>::load(row + gate + c0, g);
    Vec<T>::load(row + up + c0, u);
#pragma unroll
    for (int k = 0; k < N; ++k) g[k] = act(g[k], u[k]);
    Vec<T>::store(dst + c0, g);
    return;
  }
  for (int c = c0; c < min(c0 + N, ldo); ++c) dst[c] = from_f<T>(c < ff ? act(to_f(row[gate + c]), to_f(row[up + c])) : 0.f);
}

// ------------------------------------------------------------------------------------------------ norms and residual
// Mean and sum of squared deviations of a set, joined with another set's (every set of a merge is known, so is its count).
struct Moments {
  float n, mean, m2;
};
__device__ __forceinline__ Moments join(const Moments& a, const Moments& b) {
  const float n = a.n + b.n;
  if (n == 0.f) return a;
  const float d = b.mean - a.mean, w = b.n / n;
  return {n, a.mean + d * w, a.m2 + b.m2 + d * d * a.n * w};
}
__device__ __forceinline__ Moments join_warp(Moments m) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    Moments b;
    b.n = __shfl_xor_sync(0xffffffffu, m.n, o);
    b.mean = __shfl_xor_sync(0xffffffffu, m.mean, o);
    b.m2 = __shfl_xor_sync(0xffffffffu, m.m2, o);
    m = join(m, b);
  }
  return m;
}
// over the block; red holds 3 x 32 floats and is free again after the next barrier of the caller
__device__ __forceinline__ Moments join_block(Moments m, float* red) {
  m = join_warp(m);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) {
    red[warp] = m.n;
    red[32 + warp] = m.mean;
    red[64 + warp] = m.m2;
  }
  __syncthreads();
  Moments r = {0.f, 0.f, 0.f};
  if (lane < nw) r = {red[lane], red[32 + lane], red[64 + lane]};
  return join_warp(r);
}

// A thread owns the values c with (c / U) % threads == thread, up to R of them. VEC: U = 4, one access each; else U = 1.
template <typename T, int R, bool VEC, int THREADS>
__global__ void __launch_bounds__(THREADS) sandwich_kernel(const HySandwich a) {
  constexpr int U = VEC ? 4 : 1, G = R / U;
  __shared__ float red[3][96];
  const long long t = blockIdx.x;
  const int H = a.H, step = blockDim.x * U, first = threadIdx.x * U;
  auto each = [&](auto&& f) {  // f(register index, column)
#pragma unroll
    for (int j = 0; j < G; ++j)
      if (first + j * step < H) f(j * U, first + j * step);
  };
  auto load_f = [](const float* p, float* v) {
    if constexpr (VEC) {
      const float4 q = *reinterpret_cast<const float4*>(p);
      v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    } else {
      v[0] = p[0];
    }
  };
  auto load_w = [](const void* w, int c, float* v) {
    const T* p = static_cast<const T*>(w) + c;
    if constexpr (VEC && sizeof(T) == 2) {
      const uint2 q = *reinterpret_cast<const uint2*>(p);
      const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.x)), y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&q.y));
      v[0] = x.x; v[1] = x.y; v[2] = y.x; v[3] = y.y;
    } else if constexpr (VEC) {
      const float4 q = *reinterpret_cast<const float4*>(p);
      v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
    } else {
      v[0] = to_f(p[0]);
    }
  };
  auto moments = [&](const float (&v)[R]) {
    Moments m = {0.f, 0.f, 0.f};
    each([&](int r, int) {
#pragma unroll
      for (int k = 0; k < U; ++k) m.mean += v[r + k];
      m.n += U;
    });
    if (m.n > 0.f) m.mean /= m.n;
    each([&](int r, int) {
#pragma unroll
      for (int k = 0; k < U; ++k) m.m2 += (v[r + k] - m.mean) * (v[r + k] - m.mean);
    });
    return m;
  };
  float x[R], y[R];
  if (a.tokens) {
    int tok = a.tokens[t];
    if (tok < 0 || tok >= a.V) {
      if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, 10);
      tok = 0;
    }
    const T* row = static_cast<const T*>(a.table) + static_cast<long long>(tok) * H;
    each([&](int r, int c) { load_w(row, c, &x[r]); });
  } else {
    each([&](int r, int c) {
      load_f(a.y + t * H + c, &y[r]);
      load_f(a.x + t * H + c, &x[r]);
    });
    if (a.y2) {
      float z[R], sy = 0.f, sz = 0.f;
      each([&](int r, int c) {
        load_f(a.y2 + t * H + c, &z[r]);
#pragma unroll
        for (int k = 0; k < U; ++k) {
          sy += y[r + k] * y[r + k];
          sz += z[r + k] * z[r + k];
        }
      });
      sy = warp_sum(sy);
      sz = warp_sum(sz);
      const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
      if (lane == 0) {
        red[2][warp] = sy;
        red[2][32 + warp] = sz;
      }
      __syncthreads();
      sy = warp_sum(lane < nw ? red[2][lane] : 0.f);
      sz = warp_sum(lane < nw ? red[2][32 + lane] : 0.f);
      const float ry = 0.5f / sqrtf(sy / static_cast<float>(H) + a.eps), rz = 0.5f / sqrtf(sz / static_cast<float>(H) + a.eps);
      each([&](int r, int c) {
        float u[U], v[U];
        load_w(a.w1, c, u);
        load_w(a.w2, c, v);
#pragma unroll
        for (int k = 0; k < U; ++k) y[r + k] = y[r + k] * ry * u[k] + z[r + k] * rz * v[k];
      });
    }
    const Moments m = join_block(moments(y), red[0]);
    const float rs = 1.f / sqrtf(m.m2 / static_cast<float>(H) + a.eps);
    each([&](int r, int c) {
      float w[U];
      load_w(a.post, c, w);
#pragma unroll
      for (int k = 0; k < U; ++k) x[r + k] += (y[r + k] - m.mean) * rs * w[k];
    });
  }
  const Moments m = join_block(moments(x), red[1]);
  const float rs = 1.f / sqrtf(m.m2 / static_cast<float>(H) + a.eps);
  each([&](int r, int c) {
    float w[U];
    load_w(a.next, c, w);
    T* h = static_cast<T*>(a.h) + t * H + c;
    if constexpr (VEC) {
      *reinterpret_cast<float4*>(a.x + t * H + c) = make_float4(x[r], x[r + 1], x[r + 2], x[r + 3]);
#pragma unroll
      for (int k = 0; k < U; ++k) w[k] *= (x[r + k] - m.mean) * rs;
      if constexpr (sizeof(T) == 2) {
        const __nv_bfloat162 p = __floats2bfloat162_rn(w[0], w[1]), q = __floats2bfloat162_rn(w[2], w[3]);
        *reinterpret_cast<uint2*>(h) = make_uint2(*reinterpret_cast<const uint32_t*>(&p), *reinterpret_cast<const uint32_t*>(&q));
      } else {
        *reinterpret_cast<float4*>(h) = make_float4(w[0], w[1], w[2], w[3]);
      }
    } else {
      a.x[t * H + c] = x[r];
      h[0] = from_f<T>((x[r] - m.mean) * rs * w[0]);
    }
  });
}

template <typename T, bool VEC>
int sandwich_t(const HySandwich& a, int T_, cudaStream_t s) {
  // few rows: as many threads as a row has accesses, so that all of them are in flight at once
  const int per = VEC ? (a.H + 3) / 4 : a.H;
  auto fits = [&](int threads, int r) { return static_cast<long long>(threads) * r >= a.H; };
  if (T_ > 148 && fits(256, 32)) {
    if (fits(256, 4)) sandwich_kernel<T, 4, VEC, 256><<<T_, 256, 0, s>>>(a);
    else if (fits(256, 8)) sandwich_kernel<T, 8, VEC, 256><<<T_, 256, 0, s>>>(a);
    else if (fits(256, 16)) sandwich_kernel<T, 16, VEC, 256><<<T_, 256, 0, s>>>(a);
    else sandwich_kernel<T, 32, VEC, 256><<<T_, 256, 0, s>>>(a);
    return static_cast<int>(cudaGetLastError());
  }
  int threads = 1024;
  while (threads > 64 && threads / 2 >= per) threads /= 2;
  if (fits(threads, 4)) sandwich_kernel<T, 4, VEC, 1024><<<T_, threads, 0, s>>>(a);
  else if (fits(threads, 8)) sandwich_kernel<T, 8, VEC, 1024><<<T_, threads, 0, s>>>(a);
  else if (fits(threads, 32)) sandwich_kernel<T, 32, VEC, 1024><<<T_, threads, 0, s>>>(a);
  else return static_cast<int>(cudaErrorInvalidValue);  // wider than 32768
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int head_rows_t(const HyHeadRows& a, int T_, cudaStream_t s) {
  int per_row = 0;
  bool v2 = a.ld % 2 == 0;
  for (int i = 0; i < a.n; ++i) {
    const HyHeadOp& o = a.op[i];
    per_row += o.heads;
    v2 = v2 && (o.src | o.dim | o.col | o.pitch) % 2 == 0 && o.rot % 4 == 0 && o.ld % 2 == 0 && (reinterpret_cast<uintptr_t>(o.dst) & 7) == 0;
  }
  const long long units = static_cast<long long>(T_) * per_row;
  if (units == 0) return 0;
  const unsigned blocks = static_cast<unsigned>((units + 7) / 8);
  if (v2) head_rows_kernel<T, true><<<blocks, 256, 0, s>>>(a, per_row, units);
  else head_rows_kernel<T, false><<<blocks, 256, 0, s>>>(a, per_row, units);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int gated_act_t(const void* proj, long long ld, int gate, int up, int ff, int act, int T_, void* out, int ldo, cudaStream_t s) {
  constexpr int N = Vec<T>::N;
  const bool vec = (gate | up) % N == 0 && aligned16<T>(proj, ld) && aligned16<T>(out, ldo);
  const int per_row = (ldo + N - 1) / N;
  const long long units = static_cast<long long>(T_) * per_row;
  if (units == 0) return 0;
  const unsigned blocks = static_cast<unsigned>((units + 255) / 256);
  const T* p = static_cast<const T*>(proj);
  T* o = static_cast<T*>(out);
  if (act == 1) gated_act_kernel<T, 1><<<blocks, 256, 0, s>>>(p, ld, gate, up, ff, ldo, o, vec, units, per_row);
  else gated_act_kernel<T, 0><<<blocks, 256, 0, s>>>(p, ld, gate, up, ff, ldo, o, vec, units, per_row);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace

int hy_head_rows(bool f32, const HyHeadRows& a, int T, cudaStream_t s) { return f32 ? head_rows_t<float>(a, T, s) : head_rows_t<bf16>(a, T, s); }

int hy_gated_act(bool f32, const void* proj, long long ld, int gate, int up, int ff, int act, int T, void* out, int ldo, cudaStream_t s) {
  return f32 ? gated_act_t<float>(proj, ld, gate, up, ff, act, T, out, ldo, s) : gated_act_t<bf16>(proj, ld, gate, up, ff, act, T, out, ldo, s);
}

int hy_sandwich(bool f32, const HySandwich& a, int T, cudaStream_t s) {
  const bool vec = a.H % 4 == 0;  // (rows and weights start on 16-byte boundaries: the parameter store and the allocator align them)
  if (f32) return vec ? sandwich_t<float, true>(a, T, s) : sandwich_t<float, false>(a, T, s);
  return vec ? sandwich_t<bf16, true>(a, T, s) : sandwich_t<bf16, false>(a, T, s);
}

}  // namespace mb
