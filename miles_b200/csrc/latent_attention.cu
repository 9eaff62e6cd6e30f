// Latent attention over the paged latent cache.
//
// A cached row holds one token's latent c (rank values) and the rotated key part shared by all heads. Two forms of the same
// attention:
//  * absorbed: queries are taken into latent space (W_uk^T q), scores and outputs are products with the cached rows
//    themselves, all heads of a token reading the same bytes; W_uv brings the result back. Decoding uses it: the cache is
//    the only thing that grows with the context, and it is read once for all heads.
//  * materialised (latent_prefill.cu): keys and values of the visible range are projected once, which needs far fewer
//    operations when many queries share them. Prompts use it.
// This file has the absorbed form (tensor-core decode kernel, and a plain kernel for any sizes and for 32-bit), the query /
// output projections around it, and the row gather and query layout the materialised form starts from.
#include <float.h>

#include "hybrid.h"
#include "hybrid_common.cuh"

namespace mb {
namespace {

using namespace hy;

constexpr int TT = 8;  // rows that share the weight reads of a projection block

__device__ __forceinline__ long long row_slot(const HyLatent& a, int seq, int pos) {
  const int pg = pos / a.page_size;
  if (pg >= a.max_pages) return -1;
  const long long page = a.table[static_cast<long long>(seq) * a.max_pages + pg];
  const long long slot = page * a.page_size + pos % a.page_size;
  return (page < 0 || slot >= a.num_slots) ? -1 : slot;
}

// ------------------------------------------------------------------------------------------------ projections
// Block (x, head, row tile): x < nr: 128 latent columns; x == nr: the rotated part and the padding.
template <typename T, typename O>
__global__ void __launch_bounds__(128) absorb_q_kernel(const HyLatent a, const T* __restrict__ q, const int* __restrict__ positions,
                                                       int n_rows, O* __restrict__ ql, int qld, int nr) {
  extern __shared__ float qs[];  // [TT][dim]
  const int h = blockIdx.y, t0 = blockIdx.z * TT, qd = a.dim + a.rot;
  if (static_cast<int>(blockIdx.x) == nr) {
    for (int i = threadIdx.x; i < TT * (qld - a.rank); i += blockDim.x) {
      const int b = i / (qld - a.rank), c = i - b * (qld - a.rank), t = t0 + b;
      if (t >= n_rows) break;
      float v = 0.f;
      if (c < a.rot) {
        const T* src = q + (static_cast<long long>(t) * a.heads + h) * qd + a.dim;
        float sn, cs;
        sincosf(static_cast<float>(positions[t]) * a.freq[c >> 1], &sn, &cs);
        const float u = to_f(src[c & ~1]), w = to_f(src[c | 1]);
        v = (c & 1) ? w * cs + u * sn : u * cs - w * sn;
      }
      ql[(static_cast<long long>(t) * a.heads + h) * qld + a.rank + c] = from_f<O>(v);
    }
    return;
  }
  for (int i = threadIdx.x; i < TT * a.dim; i += blockDim.x) {
    const int b = i / a.dim, d = i - b * a.dim;
    qs[i] = t0 + b < n_rows ? to_f(q[(static_cast<long long>(t0 + b) * a.heads + h) * qd + d]) : 0.f;
  }
  __syncthreads();
  const int r = blockIdx.x * 128 + threadIdx.x;
  if (r >= a.rank) return;
  const T* w = static_cast<const T*>(a.ukv) + static_cast<long long>(h) * a.dim * a.rank + r;
  float acc[TT];
#pragma unroll
  for (int b = 0; b < TT; ++b) acc[b] = 0.f;
#pragma unroll 8
  for (int d = 0; d < a.dim; ++d) {
    const float v = to_f(w[static_cast<long long>(d) * a.rank]);
#pragma unroll
    for (int b = 0; b < TT; ++b) acc[b] += v * qs[b * a.dim + d];
  }
#pragma unroll
  for (int b = 0; b < TT; ++b)
    if (t0 + b < n_rows) ql[(static_cast<long long>(t0 + b) * a.heads + h) * qld + r] = from_f<O>(acc[b]);
}

// Block (x, head, row tile): 32 output values of a head. o is [T, heads, splits, rank] with (max, sum) per split when ml is
// given (unnormalised partial outputs), else normalised and splits = 1.
template <typename T>
__global__ void __launch_bounds__(128) latent_up_kernel(const HyLatent a, const float* __restrict__ o, const float* __restrict__ ml,
                                                        int splits, int n_rows, T* __restrict__ cat, int ldc, bool vec) {
  extern __shared__ float os[];  // [TT][rank]
  __shared__ float coef[TT][64];
  const int h = blockIdx.y, t0 = blockIdx.z * TT;
  const int rows = min(TT, n_rows - t0);
  if (ml) {
    if (static_cast<int>(threadIdx.x) < rows) {
      const float* p = ml + (static_cast<long long>(t0 + threadIdx.x) * a.heads + h) * splits * 2;
      float m = -FLT_MAX, l = 0.f;
      for (int s = 0; s < splits; ++s) m = fmaxf(m, p[2 * s]);
      for (int s = 0; s < splits; ++s) {
        const float c = p[2 * s] == -FLT_MAX ? 0.f : exp2f(p[2 * s] - m);
        coef[threadIdx.x][s] = c;
        l += c * p[2 * s + 1];
      }
      const float inv = l > 0.f ? 1.f / l : 0.f;
      for (int s = 0; s < splits; ++s) coef[threadIdx.x][s] *= inv;
    }
    __syncthreads();
  }
  for (int i = threadIdx.x; i < TT * a.rank; i += blockDim.x) {
    const int b = i / a.rank, r = i - b * a.rank;
    float v = 0.f;
    if (b < rows) {
      const float* p = o + (static_cast<long long>(t0 + b) * a.heads + h) * splits * a.rank + r;
      if (ml) {
        for (int s = 0; s < splits; ++s)
          if (coef[b][s] != 0.f) v += coef[b][s] * p[static_cast<long long>(s) * a.rank];
      } else {
        v = p[0];
      }
    }
    os[i] = v;
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* wv = static_cast<const T*>(a.ukv) + static_cast<long long>(a.heads) * a.dim * a.rank;
  const int v_end = min(a.vdim, static_cast<int>(blockIdx.x) * 32 + 32);
  for (int v = blockIdx.x * 32 + warp; v < v_end; v += 4) {
    const T* w = wv + (static_cast<long long>(h) * a.vdim + v) * a.rank;
    float acc[TT];
#pragma unroll
    for (int b = 0; b < TT; ++b) acc[b] = 0.f;
    if (vec) {
      constexpr int N = Vec<T>::N;
      for (int r = lane * N; r < a.rank; r += 32 * N) {
        float x[N];
        Vec<T>::load(w + r, x);
#pragma unroll
        for (int b = 0; b < TT; ++b)
#pragma unroll
          for (int k = 0; k < N; ++k) acc[b] += x[k] * os[b * a.rank + r + k];
      }
    } else {
      for (int r = lane; r < a.rank; r += 32) {
        const float x = to_f(w[r]);
#pragma unroll
        for (int b = 0; b < TT; ++b) acc[b] += x * os[b * a.rank + r];
      }
    }
#pragma unroll
    for (int b = 0; b < TT; ++b) {
      acc[b] = warp_sum(acc[b]);
      if (lane == 0 && b < rows) cat[static_cast<long long>(t0 + b) * ldc + h * a.vdim + v] = from_f<T>(acc[b]);
    }
  }
}

// ------------------------------------------------------------------------------------------------ plain attention
// CTA = (head, row); 4 warps stride over the visible keys, each with its own running softmax; NR * 32 >= rank.
template <typename T, int NR>
__global__ void __launch_bounds__(128) attend_kernel(const HyLatent a, const float* __restrict__ ql, int qld,
                                                     const int* __restrict__ positions, const int* __restrict__ row_seq,
                                                     float* __restrict__ out) {
  extern __shared__ float sm[];  // query [rank + rot]; later the warps' outputs [4][rank]
  __shared__ float wm[4], wl[4];
  const int h = blockIdx.x, t = blockIdx.y, K = a.rank + a.rot;
  const int seq = row_seq ? row_seq[t] : t, pos = positions[t];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float* qr = ql + (static_cast<long long>(t) * a.heads + h) * qld;
  for (int i = threadIdx.x; i < K; i += blockDim.x) sm[i] = qr[i];
  __syncthreads();
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  float m = -FLT_MAX, l = 0.f, o[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) o[i] = 0.f;
  for (int j = lo + warp; j <= pos; j += 4) {
    const long long slot = row_slot(a, seq, j);
    if (slot < 0) {
      if (lane == 0 && a.status) atomicCAS(a.status, 0, 9);
      continue;
    }
    const T* row = static_cast<const T*>(a.rows) + slot * a.width;
    float c[NR], s = 0.f;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int k = lane + 32 * i;
      c[i] = k < a.rank ? to_f(row[k]) : 0.f;
      if (k < a.rank) s += c[i] * sm[k];
    }
    for (int k = a.rank + lane; k < K; k += 32) s += to_f(row[k]) * sm[k];
    s = warp_sum(s) * a.scale;
    const float mn = fmaxf(m, s);
    const float corr = m == -FLT_MAX ? 0.f : expf(m - mn), p = expf(s - mn);
    l = l * corr + p;
    m = mn;
#pragma unroll
    for (int i = 0; i < NR; ++i) o[i] = o[i] * corr + p * c[i];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < NR; ++i)
    if (lane + 32 * i < a.rank) sm[warp * a.rank + lane + 32 * i] = o[i];
  if (lane == 0) {
    wm[warp] = m;
    wl[warp] = l;
  }
  __syncthreads();
  float gm = -FLT_MAX, gl = 0.f, c[4];
#pragma unroll
  for (int w = 0; w < 4; ++w) gm = fmaxf(gm, wm[w]);
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    c[w] = wm[w] == -FLT_MAX ? 0.f : expf(wm[w] - gm);
    gl += c[w] * wl[w];
  }
  const float inv = gl > 0.f ? 1.f / gl : 0.f;
  for (int i = threadIdx.x; i < a.rank; i += blockDim.x) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) v += c[w] * sm[w * a.rank + i];
    out[(static_cast<long long>(t) * a.heads + h) * a.rank + i] = v * inv;
  }
}

// ------------------------------------------------------------------------------------------------ tensor-core decode
constexpr int DW = 8;     // warps
constexpr int TOK = 64;   // tokens per stage
constexpr int PLD = TOK + 8;

__device__ __forceinline__ uint32_t s_u32(const void* p) { return static_cast<uint32_t>(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, int bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
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

__host__ __device__ inline int decode_k(int rank, int rot) { return (rank + rot + 31) / 32 * 32; }

// CTA = (sequence, group of MT * 16 heads, split). Scores: a warp owns 8 of the stage's 64 tokens; outputs: a warp owns an
// eighth of the latent columns. Rows of a stage are read from the cache once for all heads of the group.
template <int MT>
__global__ void __launch_bounds__(DW * 32) latent_decode_kernel(const HyLatent a, const bf16* __restrict__ ql, int qld,
                                                                const int* __restrict__ seq_lens, int splits,
                                                                float* __restrict__ po, float* __restrict__ pml) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int KP = decode_k(a.rank, a.rot), ld = KP + 8;
  bf16* Ks = reinterpret_cast<bf16*>(raw);             // [2][TOK][ld]
  bf16* Qs = Ks + 2 * TOK * ld;                        // [MT * 16][ld]
  bf16* Ps = Qs + MT * 16 * ld;                        // [MT * 16][PLD]
  float* wmax = reinterpret_cast<float*>(Ps + MT * 16 * PLD);  // [DW][MT * 16]
  float* wsum = wmax + DW * MT * 16;                   // [DW][MT * 16]
  const int b = blockIdx.x, h0 = blockIdx.y * MT * 16, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int len = seq_lens[b];
  const long long cap = static_cast<long long>(a.max_pages) * a.page_size;
  if (len < 0 || len > cap) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, 8);
    len = len < 0 ? 0 : static_cast<int>(cap);
  }
  const int lo = a.window > 0 ? max(0, len - a.window) : 0;
  int per = (len - lo + splits - 1) / splits;
  per = (per + TOK - 1) / TOK * TOK;
  const int t_lo = min(len, lo + split * per), t_hi = min(len, t_lo + per);
  const int n_ch = (t_hi - t_lo + TOK - 1) / TOK;
  const int chunks = KP / 8, wchunks = a.width / 8;

  auto issue = [&](int ch, int stage) {
    for (int i = threadIdx.x; i < TOK * chunks; i += DW * 32) {
      const int r = i / chunks, c = i - r * chunks, t = t_lo + ch * TOK + r;
      long long slot = -1;
      if (t < t_hi) {
        slot = row_slot(a, b, t);
        if (slot < 0 && c == 0 && a.status) atomicCAS(a.status, 0, 9);
      }
      const bool ok = slot >= 0 && c < wchunks;
      cp_async16(s_u32(Ks + (stage * TOK + r) * ld + c * 8), static_cast<const bf16*>(a.rows) + (ok ? slot * a.width + c * 8 : 0), ok ? 16 : 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (n_ch > 0) issue(0, 0);
  for (int i = threadIdx.x; i < MT * 16 * chunks; i += DW * 32) {
    const int r = i / chunks, c = (i - r * chunks) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h0 + r < a.heads && c < qld) v = *reinterpret_cast<const uint4*>(ql + (static_cast<long long>(b) * a.heads + h0 + r) * qld + c);
    *reinterpret_cast<uint4*>(Qs + r * ld + c) = v;
  }
  const float sl2 = a.scale * 1.4426950408889634f;
  float m_run[MT][2], l_run[MT][2], o[MT][8][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
    m_run[mt][0] = m_run[mt][1] = -FLT_MAX;
    l_run[mt][0] = l_run[mt][1] = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) o[mt][j][0] = o[mt][j][1] = o[mt][j][2] = o[mt][j][3] = 0.f;
  }
  const int NT = (a.rank + 63) / 64;      // 8-wide column tiles per warp
  const int col0 = warp * NT * 8;
  const int r0 = lane >> 2;
  for (int ch = 0; ch < n_ch; ++ch) {
    const int stage = ch & 1;
    if (ch + 1 < n_ch) {
      issue(ch + 1, stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const bf16* Kst = Ks + stage * TOK * ld;
    float sc[MT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) sc[mt][0] = sc[mt][1] = sc[mt][2] = sc[mt][3] = 0.f;
    const uint32_t kaddr = s_u32(Kst + (warp * 8 + (lane & 7)) * ld + (lane >> 3) * 8);
    const uint32_t qaddr = s_u32(Qs + (lane & 15) * ld + ((lane >> 4) << 3));
#pragma unroll 2
    for (int k0 = 0; k0 < KP; k0 += 32) {
      uint32_t kb[4];
      ldsm4(kaddr + k0 * 2, kb);
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        uint32_t qa[4];
        ldsm4(qaddr + (mt * 16 * ld + k0) * 2, qa);
        mma(sc[mt], qa, kb[0], kb[1]);
        ldsm4(qaddr + (mt * 16 * ld + k0 + 16) * 2, qa);
        mma(sc[mt], qa, kb[2], kb[3]);
      }
    }
    const int tok = t_lo + ch * TOK + warp * 8 + (lane & 3) * 2;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
      for (int e = 0; e < 4; ++e) sc[mt][e] = tok + (e & 1) < t_hi ? sc[mt][e] * sl2 : -FLT_MAX;
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float mx = fmaxf(sc[mt][2 * r], sc[mt][2 * r + 1]);
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        if ((lane & 3) == 0) wmax[warp * MT * 16 + mt * 16 + r0 + 8 * r] = mx;
      }
    }
    __syncthreads();
    float corr[MT][2];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int row = mt * 16 + r0 + 8 * r;
        float mn = m_run[mt][r];
#pragma unroll
        for (int w = 0; w < DW; ++w) mn = fmaxf(mn, wmax[w * MT * 16 + row]);
        corr[mt][r] = m_run[mt][r] == -FLT_MAX ? 0.f : exp2f(m_run[mt][r] - mn);
        m_run[mt][r] = mn;
        const float p0 = sc[mt][2 * r] == -FLT_MAX ? 0.f : exp2f(sc[mt][2 * r] - mn);
        const float p1 = sc[mt][2 * r + 1] == -FLT_MAX ? 0.f : exp2f(sc[mt][2 * r + 1] - mn);
        l_run[mt][r] = l_run[mt][r] * corr[mt][r] + p0 + p1;
        *reinterpret_cast<__nv_bfloat162*>(Ps + row * PLD + warp * 8 + (lane & 3) * 2) = __floats2bfloat162_rn(p0, p1);
      }
    __syncthreads();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        o[mt][j][0] *= corr[mt][0]; o[mt][j][1] *= corr[mt][0];
        o[mt][j][2] *= corr[mt][1]; o[mt][j][3] *= corr[mt][1];
      }
#pragma unroll
    for (int k0 = 0; k0 < TOK; k0 += 16) {
      uint32_t pa[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) ldsm4(s_u32(Ps + (mt * 16 + (lane & 15)) * PLD + k0 + ((lane >> 4) << 3)), pa[mt]);
      const bf16* vrow = Kst + (k0 + (lane & 7) + (((lane >> 3) & 1) << 3)) * ld;
#pragma unroll
      for (int jp = 0; jp < 4; ++jp) {
        if (2 * jp >= NT) break;
        const int c = col0 + jp * 16 + ((lane >> 4) << 3);
        uint32_t vb[4];
        ldsm4t(s_u32(vrow + min(c, KP - 8)), vb);  // (columns past the row end belong to tiles that are not stored)
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma(o[mt][2 * jp], pa[mt], vb[0], vb[1]);
          mma(o[mt][2 * jp + 1], pa[mt], vb[2], vb[3]);
        }
      }
    }
    __syncthreads();  // the stage is refilled next
  }
  // sums over the warps
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float l = l_run[mt][r];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      if ((lane & 3) == 0) wsum[warp * MT * 16 + mt * 16 + r0 + 8 * r] = l;
    }
  __syncthreads();
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = mt * 16 + r0 + 8 * r, h = h0 + row;
      if (h >= a.heads) continue;
      const long long base = (static_cast<long long>(b) * a.heads + h) * splits + split;
      if (warp == 0 && (lane & 3) == 0) {
        float l = 0.f;
        for (int w = 0; w < DW; ++w) l += wsum[w * MT * 16 + row];
        pml[base * 2] = m_run[mt][r];
        pml[base * 2 + 1] = l;
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const int c = col0 + j * 8 + (lane & 3) * 2;
        if (j < NT && c < a.rank) *reinterpret_cast<float2*>(po + base * a.rank + c) = make_float2(o[mt][j][2 * r], o[mt][j][2 * r + 1]);
      }
    }
}

size_t decode_smem(int MT, int rank, int rot) {
  const int ld = decode_k(rank, rot) + 8;
  return sizeof(bf16) * (static_cast<size_t>(2) * TOK * ld + MT * 16 * ld + MT * 16 * PLD) + sizeof(float) * 2 * DW * MT * 16;
}

// ------------------------------------------------------------------------------------------------ materialised form: inputs
template <typename T>
__global__ void __launch_bounds__(256) gather_rows_kernel(const HyLatent a, const int4* __restrict__ ranges, T* __restrict__ out) {
  const int4 rg = ranges[blockIdx.y];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int i = blockIdx.x * 8 + warp;
  if (i >= rg.w) return;
  const long long slot = row_slot(a, rg.x, rg.y + i);
  T* dst = out + static_cast<long long>(rg.z + i) * a.width;
  constexpr int N = 16 / sizeof(T);
  for (int c = lane * N; c < a.width; c += 32 * N) {
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (slot >= 0) v = *reinterpret_cast<const uint4*>(static_cast<const T*>(a.rows) + slot * a.width + c);
    *reinterpret_cast<uint4*>(dst + c) = v;
  }
  if (slot < 0 && lane == 0 && a.status) atomicCAS(a.status, 0, 9);
}

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
  const size_t smem = sizeof(float) * TT * a.dim;
  auto kern = absorb_q_kernel<T, O>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(nr + 1, a.heads, (n + TT - 1) / TT), 128, smem, s>>>(a, static_cast<const T*>(q), positions, n, static_cast<O*>(ql), qld, nr);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int up_t(const HyLatent& a, const float* o, const float* ml, int splits, int n, void* cat, int ldc, cudaStream_t s) {
  const size_t smem = sizeof(float) * TT * a.rank;
  auto kern = latent_up_kernel<T>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3((a.vdim + 31) / 32, a.heads, (n + TT - 1) / TT), 128, smem, s>>>(a, o, ml, splits, n, static_cast<T*>(cat), ldc,
                                                                              a.rank % Vec<T>::N == 0);
  return static_cast<int>(cudaGetLastError());
}

template <typename T>
int attend_t(const HyLatent& a, const float* ql, int qld, const int* positions, const int* row_seq, int n, float* o, cudaStream_t s) {
  const size_t smem = sizeof(float) * static_cast<size_t>(a.rank + a.rot > 4 * a.rank ? a.rank + a.rot : 4 * a.rank);
  auto go = [&](auto kern) -> int {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    kern<<<dim3(a.heads, n), 128, smem, s>>>(a, ql, qld, positions, row_seq, o);
    return static_cast<int>(cudaGetLastError());
  };
  if (a.rank <= 128) return go(attend_kernel<T, 4>);
  if (a.rank <= 256) return go(attend_kernel<T, 8>);
  if (a.rank <= 512) return go(attend_kernel<T, 16>);
  if (a.rank <= 1024) return go(attend_kernel<T, 32>);
  if (a.rank <= 2048) return go(attend_kernel<T, 64>);
  return static_cast<int>(cudaErrorInvalidValue);
}

template <int MT>
int decode_t(const HyLatent& a, const bf16* ql, int qld, const int* seq_lens, int B, int splits, float* o, float* ml, cudaStream_t s) {
  const size_t smem = decode_smem(MT, a.rank, a.rot);
  auto kern = latent_decode_kernel<MT>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  kern<<<dim3(B, (a.heads + MT * 16 - 1) / (MT * 16), splits), DW * 32, smem, s>>>(a, ql, qld, seq_lens, splits, o, ml);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace

int hy_absorb_q(bool f32, const HyLatent& a, const void* q, const int* positions, int T, void* ql, int qld, bool out_f32,
                cudaStream_t s) {
  if (f32) return absorb_t<float, float>(a, q, positions, T, ql, qld, s);
  if (out_f32) return absorb_t<bf16, float>(a, q, positions, T, ql, qld, s);
  return absorb_t<bf16, bf16>(a, q, positions, T, ql, qld, s);
}

int hy_latent_attend(bool f32, const HyLatent& a, const void* ql, int qld, const int* positions, const int* row_seq, int T,
                     float* o, cudaStream_t s) {
  const float* q = static_cast<const float*>(ql);
  return f32 ? attend_t<float>(a, q, qld, positions, row_seq, T, o, s) : attend_t<bf16>(a, q, qld, positions, row_seq, T, o, s);
}

int hy_latent_up(bool f32, const HyLatent& a, const float* o, const float* ml, int splits, int T, void* cat, int ldc, cudaStream_t s) {
  if (splits < 1 || splits > 64) return static_cast<int>(cudaErrorInvalidValue);
  return f32 ? up_t<float>(a, o, ml, splits, T, cat, ldc, s) : up_t<bf16>(a, o, ml, splits, T, cat, ldc, s);
}

bool hy_latent_decode_supported(int heads, int rank, int rot, int width) {
  return heads >= 1 && rank % 8 == 0 && rank >= 8 && rank <= 512 && width % 8 == 0 && decode_smem(heads > 16 ? 2 : 1, rank, rot) <= 227 * 1024;
}

int hy_latent_decode(const HyLatent& a, const void* ql, int qld, const int* seq_lens, int B, int splits, float* o, float* ml,
                     cudaStream_t s) {
  if (!hy_latent_decode_supported(a.heads, a.rank, a.rot, a.width) || qld % 8 != 0 || splits < 1 || splits > 64)
    return static_cast<int>(cudaErrorInvalidValue);
  const bf16* q = static_cast<const bf16*>(ql);
  return a.heads > 16 ? decode_t<2>(a, q, qld, seq_lens, B, splits, o, ml, s) : decode_t<1>(a, q, qld, seq_lens, B, splits, o, ml, s);
}

int hy_gather_rows(bool f32, const HyLatent& a, const int* ranges, int n, int max_rows, void* out, cudaStream_t s) {
  if (n <= 0 || max_rows <= 0) return 0;
  const dim3 grid((max_rows + 7) / 8, n);
  const int4* rg = reinterpret_cast<const int4*>(ranges);
  if (f32)
    gather_rows_kernel<float><<<grid, 256, 0, s>>>(a, rg, static_cast<float*>(out));
  else
    gather_rows_kernel<bf16><<<grid, 256, 0, s>>>(a, rg, static_cast<bf16*>(out));
  return static_cast<int>(cudaGetLastError());
}

int hy_pad_q(const HyLatent& a, const void* q, const int* positions, int T, int nope_pad, int rot_pad, void* out, cudaStream_t s) {
  pad_q_kernel<<<T, 256, 0, s>>>(a, static_cast<const bf16*>(q), positions, static_cast<bf16*>(out), nope_pad, rot_pad);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace mb
