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

// NH heads of a row by one warp: angles are computed once for all of them. V2: two values per access (everything even).
template <typename T, typename O, bool V2, int NH>
__device__ __forceinline__ void head_row(const HyHeadOp& op, int nh, const T* src, O* dst, float pos, float eps) {
  const int lane = threadIdx.x & 31, half = op.rot / 2;
  constexpr int W = V2 ? 2 : 1;
  float scale[NH];
#pragma unroll
  for (int k = 0; k < NH; ++k) scale[k] = op.scale;
  if (op.unit) {  // (a rotation keeps the length, so that it is measured before)
    float s[NH];
#pragma unroll
    for (int k = 0; k < NH; ++k) s[k] = 0.f;
    for (int i = lane * W; i < op.dim; i += 32 * W) {
#pragma unroll
      for (int k = 0; k < NH; ++k) {
        if (k >= nh) break;
        const T* p = src + k * op.dim + i;
        if constexpr (V2) {
          const float2 v = Pair<T>::load(p);
          s[k] += v.x * v.x + v.y * v.y;
        } else {
          s[k] += to_f(p[0]) * to_f(p[0]);
        }
      }
    }
#pragma unroll
    for (int k = 0; k < NH; ++k) scale[k] /= sqrtf(warp_sum(s[k]) / static_cast<float>(op.dim) + eps);
  }
  for (int i = lane * W; i < half; i += 32 * W) {
    float sn[W], cs[W];
#pragma unroll
    for (int k = 0; k < W; ++k) sincosf(pos * op.freq[i + k], &sn[k], &cs[k]);
    float2 u[NH], v[NH];  // all loads first: source and destination may be the same rows
#pragma unroll
    for (int k = 0; k < NH; ++k) {
      if (k >= nh) break;
      const T* p = src + k * op.dim + i;
      if constexpr (V2) {
        u[k] = Pair<T>::load(p);
        v[k] = Pair<T>::load(p + half);
      } else {
        u[k].x = to_f(p[0]);
        v[k].x = to_f(p[half]);
      }
    }
#pragma unroll
    for (int k = 0; k < NH; ++k) {
      if (k >= nh) break;
      O* d = dst + k * op.pitch + i;
      if constexpr (V2) {
        Pair<O>::store(d, make_float2((u[k].x * cs[0] - v[k].x * sn[0]) * scale[k], (u[k].y * cs[1] - v[k].y * sn[1]) * scale[k]));
        Pair<O>::store(d + half, make_float2((v[k].x * cs[0] + u[k].x * sn[0]) * scale[k], (v[k].y * cs[1] + u[k].y * sn[1]) * scale[k]));
      } else {
        d[0] = from_f<O>((u[k].x * cs[0] - v[k].x * sn[0]) * scale[k]);
        d[half] = from_f<O>((v[k].x * cs[0] + u[k].x * sn[0]) * scale[k]);
      }
    }
  }
  for (int i = op.rot + lane * W; i < op.dim; i += 32 * W) {
    float2 v[NH];
#pragma unroll
    for (int k = 0; k < NH; ++k) {
      if (k >= nh) break;
      const T* p = src + k * op.dim + i;
      if constexpr (V2) v[k] = Pair<T>::load(p);
      else v[k].x = to_f(p[0]);
    }
#pragma unroll
    for (int k = 0; k < NH; ++k) {
      if (k >= nh) break;
      O* d = dst + k * op.pitch + i;
      if constexpr (V2) Pair<O>::store(d, make_float2(v[k].x * scale[k], v[k].y * scale[k]));
      else d[0] = from_f<O>(v[k].x * scale[k]);
    }
  }
  for (int k = 0; k < nh; ++k)
    for (int i = op.dim + lane; i < op.pitch; i += 32) dst[k * op.pitch + i] = from_f<O>(0.f);
}

template <typename T, bool V2, int NH>
__global__ void __launch_bounds__(256) head_rows_kernel(const HyHeadRows a, int per_row, long long units) {
  const long long unit = static_cast<long long>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (unit >= units) return;
  const int lane = threadIdx.x & 31;
  const long long t = unit / per_row;
  int g = static_cast<int>(unit - t * per_row), o = 0;
  while (g * NH >= a.op[o].heads) g -= (a.op[o++].heads + NH - 1) / NH;
  const HyHeadOp& op = a.op[o];
  const int h = g * NH, nh = min(NH, op.heads - h);
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
  const int extra = h + nh == op.heads ? op.tail : 0;
  if (op.f32) {
    float* dst = static_cast<float*>(op.dst) + at;
    head_row<T, float, V2, NH>(op, nh, src, dst, pos, a.eps);
    for (int i = lane; i < extra; i += 32) dst[nh * op.pitch + i] = 0.f;
  } else {
    T* dst = static_cast<T*>(op.dst) + at;
    head_row<T, T, V2, NH>(op, nh, src, dst, pos, a.eps);
    for (int i = lane; i < extra; i += 32) dst[nh * op.pitch + i] = from_f<T>(0.f);
  }
}

// Many rows (bf16): the angles of a row are turned once, by a kernel in front. A head is IP lanes (a power of two) of a warp: a lane
// holds eight dimensions and their eight partners, or eight that are not rotated; a warp takes 2 * 32 / IP heads.
__global__ void __launch_bounds__(256) turns_kernel(const int* __restrict__ positions, const float* __restrict__ freq, int half, long long n,
                                                    float2* __restrict__ out) {
  const long long i = static_cast<long long>(blockIdx.x) * 256 + threadIdx.x;
  if (i >= n) return;
  const long long t = i / half;
  float sn, cs;
  sincosf(static_cast<float>(positions[t]) * freq[i - t * half], &sn, &cs);
  out[i] = make_float2(cs, sn);
}

struct HeadUnits {
  int ip[3], count[3], per_row;  // lanes of a head, units of an operation
};
__global__ void __launch_bounds__(256) head_rows8_kernel(const HyHeadRows a, const HeadUnits hu, unsigned units) {
  const unsigned unit = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (unit >= units) return;
  const int lane = threadIdx.x & 31;
  const unsigned t = unit / hu.per_row;
  int g = static_cast<int>(unit - t * hu.per_row), which = 0;
  while (g >= hu.count[which]) g -= hu.count[which++];
  const HyHeadOp& op = a.op[which];
  long long row = t;
  if (op.by_slot) {
    row = a.slots[t];
    if (row < 0 || row >= a.num_slots) {
      if (lane == 0 && a.status) atomicCAS(a.status, 0, 9);
      return;
    }
  }
  const int half = op.rot / 2, turned = half / 8, items = turned + (op.dim - op.rot) / 8, ip = hu.ip[which];
  const int item = lane & (ip - 1), per = 32 / ip;
  const bool live = item < items, pair = item < turned;
  const int c0 = pair ? item * 8 : op.rot + (item - turned) * 8;
  const bf16* src = static_cast<const bf16*>(a.proj) + t * a.ld + op.src;
  bf16* dst = static_cast<bf16*>(op.dst) + row * op.ld + op.col;
  constexpr int HN = 2;  // heads of a lane group
  const int h0 = g * per * HN + lane / ip;
  float u[HN][8], v[HN][8], cs[8], sn[8];
#pragma unroll
  for (int k = 0; k < HN; ++k) {
    const int h = h0 + k * per;
    if (h < op.heads && live) {
      Vec<bf16>::load(src + h * op.dim + c0, u[k]);
      if (pair) Vec<bf16>::load(src + h * op.dim + half + c0, v[k]);
    }
  }
  if (pair) {
    const float4* p = reinterpret_cast<const float4*>(a.turns[which] + static_cast<long long>(t) * half + c0);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float4 w = p[j];
      cs[2 * j] = w.x; sn[2 * j] = w.y;
      cs[2 * j + 1] = w.z; sn[2 * j + 1] = w.w;
    }
  }
#pragma unroll
  for (int k = 0; k < HN; ++k) {
    const int h = h0 + k * per;
    float scale = op.scale;
    if (op.unit) {
      float s = 0.f;
      if (h < op.heads && live) {
#pragma unroll
        for (int j = 0; j < 8; ++j) s += u[k][j] * u[k][j];
        if (pair) {
#pragma unroll
          for (int j = 0; j < 8; ++j) s += v[k][j] * v[k][j];
        }
      }
      for (int o = ip >> 1; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      scale *= rsqrtf(s / static_cast<float>(op.dim) + a.eps);
    }
    if (h >= op.heads) continue;
    bf16* d = dst + h * op.pitch;
    if (pair) {
      float x[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] = (u[k][j] * cs[j] - v[k][j] * sn[j]) * scale;
      Vec<bf16>::store(d + c0, x);
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] = (v[k][j] * cs[j] + u[k][j] * sn[j]) * scale;
      Vec<bf16>::store(d + half + c0, x);
    } else if (live) {
      float x[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] = u[k][j] * scale;
      Vec<bf16>::store(d + c0, x);
    }
    for (int i = op.dim + item; i < op.pitch + (h == op.heads - 1 ? op.tail : 0); i += ip) d[i] = __float2bfloat16(0.f);
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
  auto act = [](float g, float u) { return (ACT == 1 ? fmaxf(g, 0.f) : silu_t<T>(g)) * u; };
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
// Mean and sum of squared deviations of a set, joined with another set's. EVEN: both sets have n values.
struct Moments {
  float n, mean, m2;
};
__device__ __forceinline__ Moments join(const Moments& a, const Moments& b) {
  const float n = a.n + b.n;
  if (n == 0.f) return a;
  const float d = b.mean - a.mean, w = b.n / n;
  return {n, a.mean + d * w, a.m2 + b.m2 + d * d * a.n * w};
}
template <bool EVEN>
__device__ __forceinline__ Moments join_lanes(Moments m, int lanes) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    if (o >= lanes) continue;
    Moments b;
    b.mean = __shfl_xor_sync(0xffffffffu, m.mean, o);
    b.m2 = __shfl_xor_sync(0xffffffffu, m.m2, o);
    if constexpr (EVEN) {
      const float d = b.mean - m.mean;
      m.mean = 0.5f * (m.mean + b.mean);
      m.m2 = m.m2 + b.m2 + d * d * (0.5f * m.n);
      m.n *= 2.f;
    } else {
      b.n = __shfl_xor_sync(0xffffffffu, m.n, o);
      m = join(m, b);
    }
  }
  return m;
}
// over the block (a power of two of warps); red holds 3 x 32 floats and is free again after the next barrier of the caller
template <bool EVEN>
__device__ __forceinline__ Moments join_block(Moments m, float* red) {
  m = join_lanes<EVEN>(m, 32);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5, from = lane & (nw - 1);
  if (lane == 0) {
    red[warp] = m.n;
    red[32 + warp] = m.mean;
    red[64 + warp] = m.m2;
  }
  __syncthreads();
  return join_lanes<EVEN>({red[from], red[32 + from], red[64 + from]}, nw);
}

// A thread owns the values c with (c / U) % threads == thread, up to R of them. VEC: U = 4, one access each; else U = 1. EVEN: every
// thread owns R values.
template <typename T, int R, bool VEC, int THREADS, bool EVEN>
__global__ void __launch_bounds__(THREADS) sandwich_kernel(const HySandwich a) {
  constexpr int U = VEC ? 4 : 1, G = R / U;
  __shared__ float red[3][96];
  const long long t = blockIdx.x;
  const int H = a.H, step = blockDim.x * U, first = threadIdx.x * U;
  auto each = [&](auto&& f) {  // f(register index, column)
#pragma unroll
    for (int j = 0; j < G; ++j)
      if (EVEN || first + j * step < H) f(j * U, first + j * step);
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
  // weights do not depend on the reductions: where registers allow, they are fetched before them
  constexpr bool AHEAD = R <= 8;
  float wn[AHEAD ? R : 1], wp[AHEAD ? R : 1];
  if constexpr (AHEAD) {
    each([&](int r, int c) {
      load_w(a.next, c, &wn[r]);
      if (!a.tokens) load_w(a.post, c, &wp[r]);
    });
  }
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
    const Moments m = join_block<EVEN>(moments(y), red[0]);
    const float rs = 1.f / sqrtf(m.m2 / static_cast<float>(H) + a.eps);
    each([&](int r, int c) {
      float w[U];
      if constexpr (!AHEAD) load_w(a.post, c, w);
#pragma unroll
      for (int k = 0; k < U; ++k) x[r + k] += (y[r + k] - m.mean) * rs * (AHEAD ? wp[AHEAD ? r + k : 0] : w[k]);
    });
  }
  const Moments m = join_block<EVEN>(moments(x), red[1]);
  const float rs = 1.f / sqrtf(m.m2 / static_cast<float>(H) + a.eps);
  each([&](int r, int c) {
    float w[U];
    if constexpr (AHEAD) {
#pragma unroll
      for (int k = 0; k < U; ++k) w[k] = wn[r + k];
    } else {
      load_w(a.next, c, w);
    }
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

template <typename T, int R, bool VEC, int THREADS>
void sandwich_r(const HySandwich& a, int T_, int threads, cudaStream_t s) {
  if (VEC && static_cast<long long>(threads) * R == a.H) sandwich_kernel<T, R, VEC, THREADS, VEC><<<T_, threads, 0, s>>>(a);
  else sandwich_kernel<T, R, VEC, THREADS, false><<<T_, threads, 0, s>>>(a);
}

template <typename T, bool VEC>
int sandwich_t(const HySandwich& a, int T_, cudaStream_t s) {
  // few rows: as many threads as a row has accesses, so that all of them are in flight at once
  const int per = VEC ? (a.H + 3) / 4 : a.H;
  auto fits = [&](int threads, int r) { return static_cast<long long>(threads) * r >= a.H; };
  if (T_ > 148 && fits(256, 32)) {
    if (fits(256, 4)) sandwich_r<T, 4, VEC, 256>(a, T_, 256, s);
    else if (fits(256, 8)) sandwich_r<T, 8, VEC, 256>(a, T_, 256, s);
    else if (fits(256, 16)) sandwich_r<T, 16, VEC, 256>(a, T_, 256, s);
    else sandwich_r<T, 32, VEC, 256>(a, T_, 256, s);
    return static_cast<int>(cudaGetLastError());
  }
  int threads = 1024;
  while (threads > 64 && threads / 2 >= per) threads /= 2;
  if (fits(threads, 4)) sandwich_r<T, 4, VEC, 1024>(a, T_, threads, s);
  else if (fits(threads, 8)) sandwich_r<T, 8, VEC, 1024>(a, T_, threads, s);
  else if (fits(threads, 32)) sandwich_r<T, 32, VEC, 1024>(a, T_, threads, s);
  else return static_cast<int>(cudaErrorInvalidValue);  // wider than 32768
  return static_cast<int>(cudaGetLastError());
}

template <typename T, int NH>
int head_rows_nh(const HyHeadRows& a, int T_, bool v2, cudaStream_t s) {
  int per_row = 0;
  for (int i = 0; i < a.n; ++i) per_row += (a.op[i].heads + NH - 1) / NH;
  const long long units = static_cast<long long>(T_) * per_row;
  if (units == 0) return 0;
  const unsigned blocks = static_cast<unsigned>((units + 7) / 8);
  if (v2) head_rows_kernel<T, true, NH><<<blocks, 256, 0, s>>>(a, per_row, units);
  else head_rows_kernel<T, false, NH><<<blocks, 256, 0, s>>>(a, per_row, units);
  return static_cast<int>(cudaGetLastError());
}
template <typename T>
int head_rows_t(const HyHeadRows& a, int T_, cudaStream_t s) {
  bool v2 = a.ld % 2 == 0;
  for (int i = 0; i < a.n; ++i) {
    const HyHeadOp& o = a.op[i];
    v2 = v2 && (o.src | o.dim | o.col | o.pitch) % 2 == 0 && o.rot % 4 == 0 && o.ld % 2 == 0 && (reinterpret_cast<uintptr_t>(o.dst) & 7) == 0;
  }
  if constexpr (sizeof(T) == 2) {
    bool eight = aligned16<T>(a.proj, a.ld);
    for (int i = 0; i < a.n; ++i) {
      const HyHeadOp& o = a.op[i];
      eight = eight && !o.f32 && (o.src | o.dim | o.col | o.pitch) % 8 == 0 && o.rot % 16 == 0 && aligned16<T>(o.dst, o.ld) &&
              (o.dim - o.rot / 2) / 8 <= 32 && (o.rot == 0 || a.turns[i]);
    }
    if (eight) {
      for (int i = 0; i < a.n; ++i) {
        const long long n = static_cast<long long>(T_) * (a.op[i].rot / 2);
        if (a.fill[i] && n > 0)
          turns_kernel<<<static_cast<unsigned>((n + 255) / 256), 256, 0, s>>>(a.positions, a.op[i].freq, a.op[i].rot / 2, n, a.turns[i]);
      }
      HeadUnits hu = {};
      for (int i = 0; i < a.n; ++i) {
        const HyHeadOp& o = a.op[i];
        int ip = 1;
        while (ip < (o.dim - o.rot / 2) / 8) ip <<= 1;
        hu.ip[i] = ip;
        hu.count[i] = (o.heads + 64 / ip - 1) / (64 / ip);
        hu.per_row += hu.count[i];
      }
      const long long units = static_cast<long long>(T_) * hu.per_row;
      if (units > 0x7fffffffll) return static_cast<int>(cudaErrorInvalidValue);
      head_rows8_kernel<<<static_cast<unsigned>((units + 7) / 8), 256, 0, s>>>(a, hu, static_cast<unsigned>(units));
      return static_cast<int>(cudaGetLastError());
    }
  }
  return T_ > 512 ? head_rows_nh<T, 8>(a, T_, v2, s) : head_rows_nh<T, 1>(a, T_, v2, s);
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
