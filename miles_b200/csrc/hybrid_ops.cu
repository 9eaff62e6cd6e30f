// Row-wise kernels of planned layers: embedding + first norm, the tails that assemble a layer's fused output row, and the
// per-layer token input with residual update and the next norm.
//
// A parallel layer is two large products: everything that reads the normed input (mixer input | gate | up) and everything
// that writes the residual (mixer output | down). The kernels here sit between them, so that no intermediate of a layer is
// read or written twice: the tail kernels write mixer output and silu(gate) * up side by side into the row the second
// product reads, and the token-input kernel ends in the norm of the next layer.
#include <cooperative_groups.h>

#include "hybrid.h"
#include "hybrid_common.cuh"

namespace mb {
namespace {

using namespace hy;
namespace cg = cooperative_groups;

// ------------------------------------------------------------------------------------------------ embedding + norm
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) embed_norm_kernel(const int* __restrict__ tokens, const T* __restrict__ table, int V, int H,
                                                         const T* __restrict__ w, const T* __restrict__ b,
                                                         const T* __restrict__ alpha, float* __restrict__ x, T* __restrict__ h,
                                                         int* __restrict__ status) {
  const long long t = blockIdx.x;
  int tok = tokens[t];
  if (tok < 0 || tok >= V) {
    if (threadIdx.x == 0 && status) atomicCAS(status, 0, 10);
    tok = 0;
  }
  const float a = to_f(alpha[0]);
  const T* row = table + static_cast<long long>(tok) * H;
  if constexpr (VEC) {
    constexpr int N = Vec<T>::N;
    for (int c = threadIdx.x * N; c < H; c += blockDim.x * N) {
      float v[N], wv[N], bv[N], o[N];
      Vec<T>::load(row + c, v);
      Vec<T>::load(w + c, wv);
      Vec<T>::load(b + c, bv);
#pragma unroll
      for (int i = 0; i < N; ++i) o[i] = tanhf(a * v[i]) * wv[i] + bv[i];
#pragma unroll
      for (int i = 0; i < N; i += 4) *reinterpret_cast<float4*>(x + t * H + c + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
      Vec<T>::store(h + t * H + c, o);
    }
  } else {
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
      const float v = to_f(row[c]);
      x[t * H + c] = v;
      h[t * H + c] = from_f<T>(tanhf(a * v) * to_f(w[c]) + to_f(b[c]));
    }
  }
}

// ------------------------------------------------------------------------------------------------ the fused output row
// Feed-forward part and padding of row t (all threads of the block).
template <typename T>
__device__ __forceinline__ void cat_ff(const HyCat& c, long long t, bool vec) {
  const T* pr = static_cast<const T*>(c.proj) + t * c.ld;
  T* out = static_cast<T*>(c.cat) + t * c.ldc;
  const T zero = from_f<T>(0.f);
  const int ff_end = c.down + c.ff;
  for (int i = c.mixed + threadIdx.x; i < (c.ff > 0 ? c.down : c.ldc); i += blockDim.x) out[i] = zero;
  if (c.ff <= 0) return;
  for (int i = ff_end + threadIdx.x; i < c.ldc; i += blockDim.x) out[i] = zero;
  if (vec) {
    constexpr int N = Vec<T>::N;
    for (int i = threadIdx.x * N; i < c.ff; i += blockDim.x * N) {
      float g[N], u[N];
      Vec<T>::load(pr + c.gate + i, g);
      Vec<T>::load(pr + c.up + i, u);
#pragma unroll
      for (int k = 0; k < N; ++k) g[k] = silu_f(g[k]) * u[k];
      Vec<T>::store(out + c.down + i, g);
    }
  } else {
    for (int i = threadIdx.x; i < c.ff; i += blockDim.x)
      out[c.down + i] = from_f<T>(silu_f(to_f(pr[c.gate + i])) * to_f(pr[c.up + i]));
  }
}

// Grid (T, 2): y = 0 the mixer part, y = 1 the feed-forward part of a row.
template <typename T>
__global__ void __launch_bounds__(1024) mamba_tail_kernel(const T* __restrict__ y, const T* __restrict__ w, int inner, int ng, float eps,
                                                         const HyCat c, bool ff_vec, bool mix_vec) {
  const long long t = blockIdx.x;
  if (blockIdx.y == 1) {
    cat_ff<T>(c, t, ff_vec);
    return;
  }
  extern __shared__ float sm[];  // [inner] gated values, then [32] partial sums
  float* part = sm + inner;
  const T* yr = y + t * inner;
  const T* z = static_cast<const T*>(c.proj) + t * c.ld;
  T* out = static_cast<T*>(c.cat) + t * c.ldc;
  if (mix_vec) {
    constexpr int N = Vec<T>::N;
    for (int i = threadIdx.x * N; i < inner; i += blockDim.x * N) {
      float a[N], g[N];
      Vec<T>::load(yr + i, a);
      Vec<T>::load(z + i, g);
#pragma unroll
      for (int k = 0; k < N; ++k) sm[i + k] = a[k] * silu_f(g[k]);
    }
  } else {
    for (int i = threadIdx.x; i < inner; i += blockDim.x) sm[i] = to_f(yr[i]) * silu_f(to_f(z[i]));
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, size = inner / ng, nw = blockDim.x >> 5;
  const int wpg = ng >= nw ? 1 : nw / ng;  // warps per group
  for (int g0 = 0; g0 < ng; g0 += nw / wpg) {
    const int g = g0 + warp / wpg;
    const bool live = g < ng && warp < (nw / wpg) * wpg;
    float s = 0.f;
    if (live)
      for (int i = (warp % wpg) * 32 + lane; i < size; i += wpg * 32) {
        const float v = sm[g * size + i];
        s += v * v;
      }
    s = warp_sum(s);
    if (lane == 0) part[warp] = s;
    __syncthreads();
    if (live) {
      float tot = 0.f;
      for (int k = 0; k < wpg; ++k) tot += part[(warp / wpg) * wpg + k];
      const float r = 1.f / sqrtf(tot / static_cast<float>(size) + eps);
      for (int i = (warp % wpg) * 32 + lane; i < size; i += wpg * 32)
        out[g * size + i] = from_f<T>(sm[g * size + i] * r * to_f(w[g * size + i]));
    }
    __syncthreads();
  }
}

// Grid (T, 2): y = 0 the latents of a row, y = 1 its feed-forward part.
template <typename T>
__global__ void __launch_bounds__(1024) latent_in_kernel(const HyLatentIn a, const HyCat c, bool ff_vec) {
  __shared__ float red[33];
  const long long t = blockIdx.x;
  if (blockIdx.y == 1) {
    cat_ff<T>(c, t, ff_vec);
    return;
  }
  const T* pr = static_cast<const T*>(c.proj) + t * c.ld;
  float s = 0.f;
  for (int i = threadIdx.x; i < a.q_rank; i += blockDim.x) {
    const float v = to_f(pr[a.dq + i]);
    s += v * v;
  }
  float r = 1.f / sqrtf(block_sum(s, red) / static_cast<float>(a.q_rank) + a.eps);
  T* cq = static_cast<T*>(a.cq) + t * a.q_rank;
  for (int i = threadIdx.x; i < a.q_rank; i += blockDim.x)
    cq[i] = from_f<T>(to_f(pr[a.dq + i]) * r * to_f(static_cast<const T*>(a.q_norm)[i]));
  if (a.dkv < 0) return;
  const long long slot = a.slots[t];
  if (slot < 0 || slot >= a.num_slots) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, 9);
    return;
  }
  s = 0.f;
  for (int i = threadIdx.x; i < a.kv_rank; i += blockDim.x) {
    const float v = to_f(pr[a.dkv + i]);
    s += v * v;
  }
  r = 1.f / sqrtf(block_sum(s, red) / static_cast<float>(a.kv_rank) + a.eps);
  T* row = static_cast<T*>(a.rows) + slot * a.width;
  for (int i = threadIdx.x; i < a.kv_rank; i += blockDim.x)
    row[i] = from_f<T>(to_f(pr[a.dkv + i]) * r * to_f(static_cast<const T*>(a.kv_norm)[i]));
  const float pos = static_cast<float>(a.positions[t]);
  const T* kr = pr + a.dkv + a.kv_rank;
  for (int k = threadIdx.x; k < a.rot_dim / 2; k += blockDim.x) {
    float sn, cs;
    sincosf(pos * a.freq[k], &sn, &cs);
    const float u = to_f(kr[2 * k]), v = to_f(kr[2 * k + 1]);
    row[a.kv_rank + 2 * k] = from_f<T>(u * cs - v * sn);
    row[a.kv_rank + 2 * k + 1] = from_f<T>(v * cs + u * sn);
  }
  for (int i = a.kv_rank + a.rot_dim + threadIdx.x; i < a.width; i += blockDim.x) row[i] = from_f<T>(0.f);
}

// ------------------------------------------------------------------------------------------------ per-layer token input
constexpr int CS = 8;    // CTAs per cluster: each owns an eighth of the gate rows and of the output columns
constexpr int STHREADS = 1024;
constexpr int LPR = 4;   // lanes per row of the projection
constexpr int PF = 8;    // 16-byte pieces of a projection row a lane fetches ahead (rows of up to LPR * PF * 8 bf16 values)

// TB tokens per cluster. The weights do not depend on anything computed here, so their loads are issued first: the gate rows of
// the warps, and the first projection row of every group of LPR lanes.
template <typename T, int TB>
__global__ void __launch_bounds__(STHREADS) side_fused_kernel(const HySide a, int n_tok, bool vec_h, bool vec_s) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float wred[STHREADS / 32][TB];
  constexpr int N = Vec<T>::N;
  cg::cluster_group cl = cg::this_cluster();
  const int rank = static_cast<int>(cl.block_rank());
  const int t0 = static_cast<int>(blockIdx.x / CS) * TB;
  const int H = a.H, sd = a.sd;
  const int Hp = (H + 3) & ~3, sp = (sd + 3) & ~3;
  float* xs = sm;                       // [TB][Hp] residual with delta
  float* gs = xs + TB * Hp;             // [TB][sp]
  float* ss = gs + TB * sp;             // [TB][CS] partial sums of squares
  const int cols = (H + CS - 1) / CS, c0 = rank * cols, c1 = min(H, c0 + cols);
  float* ys = ss + TB * CS;             // [TB][cols]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = threadIdx.x & (LPR - 1);
  const int row_of = threadIdx.x / LPR;
  const bool ahead = vec_s && sd <= LPR * PF * N;
  uint4 pw[PF];
  if (ahead) {
    const int c = c0 + row_of;
#pragma unroll
    for (int i = 0; i < PF; ++i) {
      const int k = (i * LPR + sub) * N;
      pw[i] = make_uint4(0u, 0u, 0u, 0u);
      if (c < c1 && k < sd) pw[i] = *reinterpret_cast<const uint4*>(static_cast<const T*>(a.proj) + static_cast<long long>(c) * sd + k);
    }
  }
  for (int b = 0; b < TB; ++b) {
    const int t = t0 + b;
    for (int i = threadIdx.x; i < H; i += STHREADS) {
      float v = 0.f;
      if (t < n_tok) {
        v = a.x[static_cast<long long>(t) * H + i];
        if (a.delta) v += a.delta[static_cast<long long>(t) * H + i];
      }
      xs[b * Hp + i] = v;
    }
  }
  cl.sync();  // every CTA of the cluster runs before its shared memory is written from another
  // gate products of this CTA's rows, sent to every CTA of the cluster
  const int dims = (sd + CS - 1) / CS, d0 = rank * dims, d1 = min(sd, d0 + dims);
  for (int d = d0 + warp; d < d1; d += STHREADS / 32) {
    const T* w = static_cast<const T*>(a.gate) + static_cast<long long>(d) * H;
    float s[TB];
#pragma unroll
    for (int b = 0; b < TB; ++b) s[b] = 0.f;
    if (vec_h) {
#pragma unroll 4
      for (int i = lane * N; i < H; i += 32 * N) {
        float v[N];
        Vec<T>::load(w + i, v);
#pragma unroll
        for (int b = 0; b < TB; ++b)
#pragma unroll
          for (int k = 0; k < N; k += 4) {
            const float4 x = *reinterpret_cast<const float4*>(xs + b * Hp + i + k);
            s[b] += v[k] * x.x + v[k + 1] * x.y + v[k + 2] * x.z + v[k + 3] * x.w;
          }
      }
    } else {
      for (int i = lane; i < H; i += 32) {
        const float v = to_f(w[i]);
#pragma unroll
        for (int b = 0; b < TB; ++b) s[b] += v * xs[b * Hp + i];
      }
    }
#pragma unroll
    for (int b = 0; b < TB; ++b) {
      s[b] = warp_sum(s[b]);
      const int t = t0 + b;
      float g = 0.f;
      if (t < n_tok) {
        int tok = a.tokens[t];
        if (tok < 0 || tok >= a.V) {
          if (lane == 0 && a.status) atomicCAS(a.status, 0, 10);
          tok = 0;
        }
        const float e = to_f(static_cast<const T*>(a.embed)[static_cast<long long>(tok) * a.embed_ld + a.embed_col + d]);
        g = to_f(from_f<T>(gelu_tanh_f(s[b]) * e));
      }
      if (lane < CS) *cl.map_shared_rank(gs + b * sp + d, lane) = g;
    }
  }
  cl.sync();
  // this CTA's output columns: LPR lanes per row of the projection
  float sq[TB];
#pragma unroll
  for (int b = 0; b < TB; ++b) sq[b] = 0.f;
  for (int base = c0; base < c1; base += STHREADS / LPR) {
    const int c = base + row_of;
    const T* w = static_cast<const T*>(a.proj) + static_cast<long long>(c) * sd;
    float s[TB];
#pragma unroll
    for (int b = 0; b < TB; ++b) s[b] = 0.f;
    auto dot = [&](const uint4& raw, int k) {
      float v[N];
      Vec<T>::load(reinterpret_cast<const T*>(&raw), v);
#pragma unroll
      for (int b = 0; b < TB; ++b)
#pragma unroll
        for (int j = 0; j < N; j += 4) {
          const float4 g = *reinterpret_cast<const float4*>(gs + b * sp + k + j);
          s[b] += v[j] * g.x + v[j + 1] * g.y + v[j + 2] * g.z + v[j + 3] * g.w;
        }
    };
    if (ahead) {
#pragma unroll
      for (int i = 0; i < PF; ++i)
        if ((i * LPR + sub) * N < sd) dot(pw[i], (i * LPR + sub) * N);
      const int cn = c + STHREADS / LPR;  // the next row of this lane
#pragma unroll
      for (int i = 0; i < PF; ++i) {
        const int k = (i * LPR + sub) * N;
        if (cn < c1 && k < sd) pw[i] = *reinterpret_cast<const uint4*>(static_cast<const T*>(a.proj) + static_cast<long long>(cn) * sd + k);
      }
    } else if (c < c1) {
      if (vec_s) {
        for (int k = sub * N; k < sd; k += LPR * N) dot(*reinterpret_cast<const uint4*>(w + k), k);
      } else {
        for (int i = sub; i < sd; i += LPR) {
          const float v = to_f(w[i]);
#pragma unroll
          for (int b = 0; b < TB; ++b) s[b] += v * gs[b * sp + i];
        }
      }
    }
#pragma unroll
    for (int b = 0; b < TB; ++b) {
      s[b] += __shfl_xor_sync(0xffffffffu, s[b], 1);
      s[b] += __shfl_xor_sync(0xffffffffu, s[b], 2);
      if (c < c1 && sub == 0) {
        ys[b * cols + c - c0] = s[b];
        sq[b] += s[b] * s[b];
      }
    }
  }
#pragma unroll
  for (int b = 0; b < TB; ++b) {
    sq[b] = warp_sum(sq[b]);
    if (lane == 0) wred[warp][b] = sq[b];
  }
  __syncthreads();
  if (warp < TB) {
    const float tot = warp_sum(wred[lane][warp]);
    if (lane < CS) *cl.map_shared_rank(ss + warp * CS + rank, lane) = tot;
  }
  cl.sync();
  const float al = to_f(static_cast<const T*>(a.na)[0]);
  for (int b = 0; b < TB; ++b) {
    const int t = t0 + b;
    if (t >= n_tok) break;
    float tot = 0.f;
#pragma unroll
    for (int k = 0; k < CS; ++k) tot += ss[b * CS + k];
    const float r = 1.f / sqrtf(tot / static_cast<float>(H) + a.eps);
    for (int c = c0 + threadIdx.x; c < c1; c += STHREADS) {
      const float v = xs[b * Hp + c] + ys[b * cols + c - c0] * r * to_f(static_cast<const T*>(a.norm)[c]);
      a.x[static_cast<long long>(t) * H + c] = v;
      static_cast<T*>(a.h)[static_cast<long long>(t) * H + c] =
          from_f<T>(tanhf(al * v) * to_f(static_cast<const T*>(a.nw)[c]) + to_f(static_cast<const T*>(a.nb)[c]));
    }
  }
}

__global__ void __launch_bounds__(256) cast_rows_kernel(float* __restrict__ x, const float* __restrict__ delta, bf16* __restrict__ o,
                                                        long long n) {
  const long long i = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) * 8;
  if (i + 8 <= n) {
    float4 a = *reinterpret_cast<const float4*>(x + i), b = *reinterpret_cast<const float4*>(x + i + 4);
    if (delta) {
      const float4 u = *reinterpret_cast<const float4*>(delta + i), v = *reinterpret_cast<const float4*>(delta + i + 4);
      a.x += u.x; a.y += u.y; a.z += u.z; a.w += u.w;
      b.x += v.x; b.y += v.y; b.z += v.z; b.w += v.w;
      *reinterpret_cast<float4*>(x + i) = a;
      *reinterpret_cast<float4*>(x + i + 4) = b;
    }
    const float v[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
    Vec<bf16>::store(o + i, v);
  } else {
    for (long long k = i; k < n; ++k) {
      if (delta) x[k] += delta[k];
      o[k] = __float2bfloat16(x[k]);
    }
  }
}

// V values per thread (V = 1: any width)
template <typename T, int V>
__global__ void __launch_bounds__(256) side_gate_kernel(const float* __restrict__ z, const HySide a, T* __restrict__ g, long long n) {
  const long long i = (static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x) * V;
  if (i >= n) return;
  const long long t = i / a.sd;
  const int d = static_cast<int>(i - t * a.sd);
  int tok = a.tokens[t];
  if (tok < 0 || tok >= a.V) {
    if (a.status) atomicCAS(a.status, 0, 10);
    tok = 0;
  }
  const T* e = static_cast<const T*>(a.embed) + static_cast<long long>(tok) * a.embed_ld + a.embed_col + d;
  if constexpr (V > 1) {
    float ev[V], o[V];
    Vec<T>::load(e, ev);
#pragma unroll
    for (int k = 0; k < V; k += 4) {
      const float4 v = *reinterpret_cast<const float4*>(z + i + k);
      o[k] = gelu_tanh_f(v.x) * ev[k];
      o[k + 1] = gelu_tanh_f(v.y) * ev[k + 1];
      o[k + 2] = gelu_tanh_f(v.z) * ev[k + 2];
      o[k + 3] = gelu_tanh_f(v.w) * ev[k + 3];
    }
    Vec<T>::store(g + i, o);
  } else {
    g[i] = from_f<T>(gelu_tanh_f(z[i]) * to_f(e[0]));
  }
}

template <typename T>
__global__ void __launch_bounds__(256) side_finish_kernel(const float* __restrict__ y, const HySide a, bool vec) {
  __shared__ float red[33];
  const long long t = blockIdx.x;
  const int H = a.H;
  const float* yr = y + t * H;
  float* xr = a.x + t * H;
  T* hr = static_cast<T*>(a.h) + t * H;
  const T *nw = static_cast<const T*>(a.nw), *nb = static_cast<const T*>(a.nb), *sn = static_cast<const T*>(a.norm);
  const float al = to_f(static_cast<const T*>(a.na)[0]);
  float s = 0.f;
  if (vec) {
    for (int c = threadIdx.x * 4; c < H; c += blockDim.x * 4) {
      const float4 v = *reinterpret_cast<const float4*>(yr + c);
      s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int c = threadIdx.x; c < H; c += blockDim.x) s += yr[c] * yr[c];
  }
  const float r = 1.f / sqrtf(block_sum(s, red) / static_cast<float>(H) + a.eps);
  if (vec) {
    constexpr int N = Vec<T>::N;
    for (int c = threadIdx.x * N; c < H; c += blockDim.x * N) {
      float yv[N], xv[N], w[N], b[N], q[N];
#pragma unroll
      for (int i = 0; i < N; i += 4) {
        const float4 u = *reinterpret_cast<const float4*>(yr + c + i), v = *reinterpret_cast<const float4*>(xr + c + i);
        yv[i] = u.x; yv[i + 1] = u.y; yv[i + 2] = u.z; yv[i + 3] = u.w;
        xv[i] = v.x; xv[i + 1] = v.y; xv[i + 2] = v.z; xv[i + 3] = v.w;
      }
      Vec<T>::load(sn + c, q);
      Vec<T>::load(nw + c, w);
      Vec<T>::load(nb + c, b);
#pragma unroll
      for (int i = 0; i < N; ++i) {
        xv[i] += yv[i] * r * q[i];
        w[i] = tanhf(al * xv[i]) * w[i] + b[i];
      }
#pragma unroll
      for (int i = 0; i < N; i += 4) *reinterpret_cast<float4*>(xr + c + i) = make_float4(xv[i], xv[i + 1], xv[i + 2], xv[i + 3]);
      Vec<T>::store(hr + c, w);
    }
  } else {
    for (int c = threadIdx.x; c < H; c += blockDim.x) {
      const float v = xr[c] + yr[c] * r * to_f(sn[c]);
      xr[c] = v;
      hr[c] = from_f<T>(tanhf(al * v) * to_f(nw[c]) + to_f(nb[c]));
    }
  }
}

template <typename T, int TB>
int launch_side(const HySide& a, int n_tok, cudaStream_t s) {
  const int cols = (a.H + CS - 1) / CS;
  const size_t smem = sizeof(float) * (static_cast<size_t>(TB) * (((a.H + 3) & ~3) + ((a.sd + 3) & ~3) + CS + cols));
  auto kern = side_fused_kernel<T, TB>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(static_cast<unsigned>((n_tok + TB - 1) / TB * CS));
  cfg.blockDim = dim3(STHREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = CS;
  at[0].val.clusterDim.y = at[0].val.clusterDim.z = 1;
  cfg.attrs = at;
  cfg.numAttrs = 1;
  const bool vh = a.H % Vec<T>::N == 0 && aligned16<T>(a.gate, a.H), vs = a.sd % Vec<T>::N == 0 && aligned16<T>(a.proj, a.sd);
  return static_cast<int>(cudaLaunchKernelEx(&cfg, kern, a, n_tok, vh, vs));
}

template <typename T>
bool ff_vec_ok(const HyCat& c) {
  constexpr int N = Vec<T>::N;
  return c.ff % N == 0 && c.gate % N == 0 && c.up % N == 0 && c.down % N == 0 && aligned16<T>(c.proj, c.ld) && aligned16<T>(c.cat, c.ldc);
}

template <typename T>
int embed_norm_t(const int* tokens, int T_, const void* table, int V, int H, const void* w, const void* b, const void* alpha,
                 float* x, void* h, int* status, cudaStream_t s) {
  const bool vec = H % Vec<T>::N == 0 && aligned16<T>(table, H) && aligned16<T>(w, 0) && aligned16<T>(b, 0);
  auto kern = vec ? embed_norm_kernel<T, true> : embed_norm_kernel<T, false>;
  kern<<<T_, 256, 0, s>>>(tokens, static_cast<const T*>(table), V, H, static_cast<const T*>(w), static_cast<const T*>(b),
                          static_cast<const T*>(alpha), x, static_cast<T*>(h), status);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int mamba_tail_t(const void* y, const void* w, int inner, int ng, float eps, const HyCat& c, int T_, cudaStream_t s) {
  const size_t smem = sizeof(float) * (static_cast<size_t>(inner) + 32);
  auto kern = mamba_tail_kernel<T>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  const bool mv = inner % Vec<T>::N == 0 && aligned16<T>(y, inner) && aligned16<T>(c.proj, c.ld);
  // few rows: latency counts, so every load of a row is in flight at once
  kern<<<dim3(T_, 2), T_ <= 148 ? 1024 : 256, smem, s>>>(static_cast<const T*>(y), static_cast<const T*>(w), inner, ng, eps, c, ff_vec_ok<T>(c), mv);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace

int hy_embed_norm(bool f32, const int* tokens, int T, const void* table, int V, int H, const void* w, const void* b,
                  const void* alpha, float* x, void* h, int* status, cudaStream_t s) {
  return f32 ? embed_norm_t<float>(tokens, T, table, V, H, w, b, alpha, x, h, status, s)
             : embed_norm_t<bf16>(tokens, T, table, V, H, w, b, alpha, x, h, status, s);
}

int hy_mamba_tail(bool f32, const void* y, const void* w, int inner, int norm_groups, float eps, const HyCat& c, int T,
                  cudaStream_t s) {
  return f32 ? mamba_tail_t<float>(y, w, inner, norm_groups, eps, c, T, s) : mamba_tail_t<bf16>(y, w, inner, norm_groups, eps, c, T, s);
}

int hy_latent_in(bool f32, const HyLatentIn& a, const HyCat& c, int T, cudaStream_t s) {
  if (f32)
    latent_in_kernel<float><<<dim3(T, 2), T <= 148 ? 1024 : 256, 0, s>>>(a, c, ff_vec_ok<float>(c));
  else
    latent_in_kernel<bf16><<<dim3(T, 2), T <= 148 ? 1024 : 256, 0, s>>>(a, c, ff_vec_ok<bf16>(c));
  return static_cast<int>(cudaGetLastError());
}

int hy_side_fused(bool f32, const HySide& a, int T, cudaStream_t s) {
  // tokens share the weight reads of their cluster; few rows are spread over more clusters, and wide rows bound the memory
  const bool four = T > 16 && static_cast<long long>(a.H) * 4 * 4 * 9 / 8 + a.sd * 16 < 200 * 1024;
  if (f32) return four ? launch_side<float, 4>(a, T, s) : launch_side<float, 1>(a, T, s);
  return four ? launch_side<bf16, 4>(a, T, s) : launch_side<bf16, 1>(a, T, s);
}

int hy_cast_rows(float* x, const float* delta, void* out, long long n, cudaStream_t s) {
  const long long blocks = (n + 2047) / 2048;
  cast_rows_kernel<<<static_cast<unsigned>(blocks), 256, 0, s>>>(x, delta, static_cast<bf16*>(out), n);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
static int side_gate_t(const float* z, const HySide& a, void* g, int rows, cudaStream_t s) {
  const long long n = static_cast<long long>(rows) * a.sd;
  constexpr int V = hy::Vec<T>::N;
  if (a.sd % V == 0 && a.embed_ld % V == 0)
    side_gate_kernel<T, V><<<static_cast<unsigned>((n / V + 255) / 256), 256, 0, s>>>(z, a, static_cast<T*>(g), n);
  else
    side_gate_kernel<T, 1><<<static_cast<unsigned>((n + 255) / 256), 256, 0, s>>>(z, a, static_cast<T*>(g), n);
  return static_cast<int>(cudaGetLastError());
}

int hy_side_gate(bool f32, const float* z, const HySide& a, void* g, int T, cudaStream_t s) {
  return f32 ? side_gate_t<float>(z, a, g, T, s) : side_gate_t<bf16>(z, a, g, T, s);
}

int hy_side_finish(bool f32, const float* y, const HySide& a, int T, cudaStream_t s) {
  if (f32)
    side_finish_kernel<float><<<T, 256, 0, s>>>(y, a, a.H % 8 == 0);
  else
    side_finish_kernel<bf16><<<T, 256, 0, s>>>(y, a, a.H % 8 == 0);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace mb
