// Attention over paged cache rows, whatever a row holds: a HyAttend says which columns are a head's key and which its value. Latent
// attention reads one row for all heads (keys = the whole row, values = its first columns); grouped-query attention has key and
// value columns per key head. Softmax, optionally over a sliding window, optionally with a sink (one more term per head in the
// denominator, without key or value).
//  * a plain kernel for any sizes, prompts and decoding, bf16 and 32-bit;
//  * tensor-core decoding, one row per sequence, keys split over CTAs, and the merge of the splits;
//  * the gather of visible rows from which the tcgen05 prompt attention (cached_prefill.cu) starts.
#include <float.h>

#include "hybrid.h"
#include "hybrid_mma.cuh"

namespace mb {
namespace {

using namespace hy;

__device__ __forceinline__ long long row_slot(const HyCache& a, int seq, int pos) {
  const int pg = pos / a.page_size;
  if (pg >= a.max_pages) return -1;
  const long long page = a.table[static_cast<long long>(seq) * a.max_pages + pg];
  const long long slot = page * a.page_size + pos % a.page_size;
  return (page < 0 || slot >= a.num_slots) ? -1 : slot;
}

// ------------------------------------------------------------------------------------------------ plain attention
// CTA = (head, row); 4 warps stride over the visible keys, each with its own running softmax; NR * 32 >= vd. The result goes to
// out [T, heads, vd] (fp32) or to rows of out_t (pitch ldc).
template <typename T, int NR>
__global__ void __launch_bounds__(128) attend_kernel(const HyAttend a, const float* __restrict__ ql, int qld,
                                                     const int* __restrict__ positions, const int* __restrict__ row_seq,
                                                     float* __restrict__ out, T* __restrict__ out_t, int ldc) {
  extern __shared__ float sm[];  // query [kd]; later the warps' outputs [4][vd]
  __shared__ float wm[4], wl[4];
  const int h = blockIdx.x, t = blockIdx.y, K = a.kd, g = h / a.group;
  const int kc = a.k_col + g * a.k_step, vc = a.v_col + g * a.v_step;
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
      c[i] = k < a.vd ? to_f(row[vc + k]) : 0.f;
    }
    for (int k = lane; k < K; k += 32) s += to_f(row[kc + k]) * sm[k];
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
    if (lane + 32 * i < a.vd) sm[warp * a.vd + lane + 32 * i] = o[i];
  if (lane == 0) {
    wm[warp] = m;
    wl[warp] = l;
  }
  __syncthreads();
  float gm = -FLT_MAX, gl = 0.f, c[4];
  if (a.sink) gm = to_f(static_cast<const T*>(a.sink)[h]);
#pragma unroll
  for (int w = 0; w < 4; ++w) gm = fmaxf(gm, wm[w]);
#pragma unroll
  for (int w = 0; w < 4; ++w) {
    c[w] = wm[w] == -FLT_MAX ? 0.f : expf(wm[w] - gm);
    gl += c[w] * wl[w];
  }
  if (a.sink) gl += expf(to_f(static_cast<const T*>(a.sink)[h]) - gm);
  const float inv = gl > 0.f ? 1.f / gl : 0.f;
  for (int i = threadIdx.x; i < a.vd; i += blockDim.x) {
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) v += c[w] * sm[w * a.vd + i];
    if (out) out[(static_cast<long long>(t) * a.heads + h) * a.vd + i] = v * inv;
    else out_t[static_cast<long long>(t) * ldc + h * a.vd + i] = from_f<T>(v * inv);
  }
}

// ------------------------------------------------------------------------------------------------ tensor-core decode
constexpr int DW = 8;     // warps
constexpr int TOK = 64;   // tokens per stage
constexpr int PLD = TOK + 8;

// shared columns of a row: keys padded to 32, then values padded to 16 (none of their own where they are the key's first columns)
__host__ __device__ inline bool same_columns(const HyAttend& a) { return a.v_col == a.k_col && a.v_step == a.k_step && a.vd <= a.kd; }
__host__ __device__ inline int key_cols(const HyAttend& a) { return (a.kd + 31) / 32 * 32; }
__host__ __device__ inline int row_cols(const HyAttend& a) { return key_cols(a) + (same_columns(a) ? 0 : (a.vd + 15) / 16 * 16); }

// CTA = (sequence, up to MT * 16 query heads of one key head, split). Warp (wm, wt): head tile wm; scores of the wt-th token group,
// outputs of the wt-th group of value columns. Rows of a stage are read from the cache once for all heads of the group; queries
// stay in registers (as far as they fit: the first QI of KI chunks of 32), so that shared memory carries little more than the rows.
// NTM: 8-wide output tiles per warp at most.
template <int MT, int KI, int QI, int NTM>
__global__ void __launch_bounds__(DW * 32) cached_decode_kernel(const HyAttend a, const bf16* __restrict__ ql, int qld,
                                                                const int* __restrict__ seq_lens, int splits,
                                                                float* __restrict__ po, float* __restrict__ pml) {
  constexpr int NG = DW / MT;           // token groups, column groups
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ int slot_s[2][TOK];
  const int KP = key_cols(a), cols = row_cols(a), ld = cols + 8, v0 = same_columns(a) ? 0 : KP, v_end = (same_columns(a) ? KP : cols) - 8;
  bf16* Ks = reinterpret_cast<bf16*>(raw);             // [2][TOK][ld]
  bf16* Qs = Ks + 2 * TOK * ld;                        // [MT * 16][KP + 8]
  bf16* Ps = Qs + MT * 16 * (KP + 8);                  // [MT * 16][PLD]
  float* wmax = reinterpret_cast<float*>(Ps + MT * 16 * PLD);  // [NG][MT * 16]
  float* wsum = wmax + DW * MT * 16;                   // [NG][MT * 16]
  const int per = (a.group + MT * 16 - 1) / (MT * 16), g = blockIdx.y / per;  // CTAs of a key head
  const int b = blockIdx.x, h0 = g * a.group + (blockIdx.y - g * per) * MT * 16, h1 = (g + 1) * a.group, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int wm = warp % MT, wt = warp / MT;
  int len = seq_lens[b];
  const long long cap = static_cast<long long>(a.max_pages) * a.page_size;
  if (len < 0 || len > cap) {
    if (threadIdx.x == 0 && a.status) atomicCAS(a.status, 0, 8);
    len = len < 0 ? 0 : static_cast<int>(cap);
  }
  const int lo = a.window > 0 ? max(0, len - a.window) : 0;
  int share = (len - lo + splits - 1) / splits;
  share = (share + TOK - 1) / TOK * TOK;
  const int t_lo = min(len, lo + split * share), t_hi = min(len, t_lo + share);
  const int n_ch = (t_hi - t_lo + TOK - 1) / TOK;
  const int kchunks = KP / 8, chunks = cols / 8;
  const int kc = a.k_col + g * a.k_step, vc = a.v_col + g * a.v_step;

  auto find_slots = [&](int ch) {  // by the first TOK threads, a barrier before they are used
    if (threadIdx.x >= TOK || ch >= n_ch) return;
    const int t = t_lo + ch * TOK + static_cast<int>(threadIdx.x);
    long long slot = -1;
    if (t < t_hi) {
      slot = row_slot(a, b, t);
      if (slot < 0 && a.status) atomicCAS(a.status, 0, 9);
    }
    slot_s[ch & 1][threadIdx.x] = static_cast<int>(slot);
  };
  auto issue = [&](int ch, int stage) {
#pragma unroll 2
    for (int r = warp; r < TOK; r += DW) {
      const int slot = slot_s[ch & 1][r];
      const bf16* src = static_cast<const bf16*>(a.rows) + static_cast<long long>(slot < 0 ? 0 : slot) * a.width;
      const uint32_t dst = s_u32(Ks + (stage * TOK + r) * ld);
      for (int c = lane; c < chunks; c += 32) {
        const int at = c < kchunks ? c * 8 : (c - kchunks) * 8;
        const bool ok = slot >= 0 && at < (c < kchunks ? a.kd : a.vd);
        cp16(dst + c * 16, src + (ok ? (c < kchunks ? kc : vc) + at : 0), ok ? 16 : 0);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  find_slots(0);
  for (int r = warp; r < MT * 16; r += DW)
    for (int c = lane * 8; c < KP; c += 256) {
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (h0 + r < h1 && c < qld) v = *reinterpret_cast<const uint4*>(ql + (static_cast<long long>(b) * a.heads + h0 + r) * qld + c);
      *reinterpret_cast<uint4*>(Qs + r * (KP + 8) + c) = v;
    }
  __syncthreads();
  if (n_ch > 0) issue(0, 0);
  find_slots(1);
  const uint32_t qaddr = s_u32(Qs + (wm * 16 + (lane & 15)) * (KP + 8) + ((lane >> 4) << 3));
  uint32_t qa[QI][2][4];
#pragma unroll
  for (int i = 0; i < QI; ++i)
    if (i * 32 < KP) {
      ldsm4(qaddr + i * 64, qa[i][0]);
      ldsm4(qaddr + i * 64 + 32, qa[i][1]);
    }
  const float sl2 = a.scale * 1.4426950408889634f;
  float m_run[2] = {-FLT_MAX, -FLT_MAX}, l_run[2] = {0.f, 0.f}, o[NTM][4];
#pragma unroll
  for (int j = 0; j < NTM; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  const int NT = (a.vd + 8 * NG - 1) / (8 * NG);  // 8-wide column tiles per warp
  const int col0 = wt * NT * 8;
  const int r0 = lane >> 2;
  __syncthreads();  // slots of the second stage
  for (int ch = 0; ch < n_ch; ++ch) {
    const int stage = ch & 1;
    if (ch + 1 < n_ch) {
      issue(ch + 1, stage ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    find_slots(ch + 2);  // (the ones of chunk ch have been used)
    const bf16* Kst = Ks + stage * TOK * ld;
    float sc[MT][4];
#pragma unroll
    for (int nt = 0; nt < MT; ++nt) sc[nt][0] = sc[nt][1] = sc[nt][2] = sc[nt][3] = 0.f;
    const uint32_t kaddr = s_u32(Kst + (wt * 8 * MT + (lane & 7)) * ld + (lane >> 3) * 8);
#pragma unroll
    for (int i = 0; i < KI; ++i) {
      if (i * 32 >= KP) break;
      uint32_t q0[4], q1[4];
      if (i < QI) {
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          q0[k] = qa[i < QI ? i : 0][0][k];
          q1[k] = qa[i < QI ? i : 0][1][k];
        }
      } else {
        ldsm4(qaddr + i * 64, q0);
        ldsm4(qaddr + i * 64 + 32, q1);
      }
#pragma unroll
      for (int nt = 0; nt < MT; ++nt) {
        uint32_t kb[4];
        ldsm4(kaddr + (nt * 8 * ld + i * 32) * 2, kb);
        mma(sc[nt], q0, kb[0], kb[1]);
        mma(sc[nt], q1, kb[2], kb[3]);
      }
    }
    const int tok = t_lo + ch * TOK + wt * 8 * MT + (lane & 3) * 2;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      float mx = -FLT_MAX;
#pragma unroll
      for (int nt = 0; nt < MT; ++nt)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float& v = sc[nt][2 * r + e];
          v = tok + nt * 8 + e < t_hi ? v * sl2 : -FLT_MAX;
          mx = fmaxf(mx, v);
        }
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
      mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
      if ((lane & 3) == 0) wmax[wt * MT * 16 + wm * 16 + r0 + 8 * r] = mx;
    }
    __syncthreads();
    float corr[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = wm * 16 + r0 + 8 * r;
      float mn = m_run[r];
#pragma unroll
      for (int w = 0; w < NG; ++w) mn = fmaxf(mn, wmax[w * MT * 16 + row]);
      corr[r] = m_run[r] == -FLT_MAX ? 0.f : exp2f(m_run[r] - mn);
      m_run[r] = mn;
      l_run[r] *= corr[r];
#pragma unroll
      for (int nt = 0; nt < MT; ++nt) {
        const float p0 = sc[nt][2 * r] == -FLT_MAX ? 0.f : exp2f(sc[nt][2 * r] - mn);
        const float p1 = sc[nt][2 * r + 1] == -FLT_MAX ? 0.f : exp2f(sc[nt][2 * r + 1] - mn);
        l_run[r] += p0 + p1;
        *reinterpret_cast<__nv_bfloat162*>(Ps + row * PLD + (wt * MT + nt) * 8 + (lane & 3) * 2) = __floats2bfloat162_rn(p0, p1);
      }
    }
    __syncthreads();
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int j = 0; j < NTM; ++j) {
        o[j][0] *= corr[0]; o[j][1] *= corr[0];
        o[j][2] *= corr[1]; o[j][3] *= corr[1];
      }
    }
#pragma unroll
    for (int k0 = 0; k0 < TOK; k0 += 16) {
      uint32_t pa[4];
      ldsm4(s_u32(Ps + (wm * 16 + (lane & 15)) * PLD + k0 + ((lane >> 4) << 3)), pa);
      const uint32_t vrow = s_u32(Kst + (k0 + (lane & 7) + (((lane >> 3) & 1) << 3)) * ld);
#pragma unroll
      for (int jp = 0; jp < NTM / 2; ++jp) {
        if (2 * jp >= NT) break;
        const int c = col0 + jp * 16 + ((lane >> 4) << 3);
        uint32_t vb[4];
        ldsm4t(vrow + min(v0 + c, v_end) * 2, vb);  // (columns past the row end belong to tiles that are not stored)
        mma(o[2 * jp], pa, vb[0], vb[1]);
        mma(o[2 * jp + 1], pa, vb[2], vb[3]);
      }
    }
    __syncthreads();  // the stage is refilled next
  }
  // sums over the token groups
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    float l = l_run[r];
    l += __shfl_xor_sync(0xffffffffu, l, 1);
    l += __shfl_xor_sync(0xffffffffu, l, 2);
    if ((lane & 3) == 0) wsum[wt * MT * 16 + wm * 16 + r0 + 8 * r] = l;
  }
  __syncthreads();
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = wm * 16 + r0 + 8 * r, h = h0 + row;
    if (h >= h1) continue;
    const long long base = (static_cast<long long>(b) * a.heads + h) * splits + split;
    if (wt == 0 && (lane & 3) == 0) {
      float l = 0.f;
      for (int w = 0; w < NG; ++w) l += wsum[w * MT * 16 + row];
      pml[base * 2] = m_run[r];
      pml[base * 2 + 1] = l;
    }
#pragma unroll
    for (int j = 0; j < NTM; ++j) {
      const int c = col0 + j * 8 + (lane & 3) * 2;
      if (j < NT && c < a.vd) *reinterpret_cast<float2*>(po + base * a.vd + c) = make_float2(o[j][2 * r], o[j][2 * r + 1]);
    }
  }
}

size_t decode_smem(int MT, const HyAttend& a) {
  return sizeof(bf16) * (static_cast<size_t>(2) * TOK * (row_cols(a) + 8) + MT * 16 * (key_cols(a) + 8) + MT * 16 * PLD) + sizeof(float) * 2 * DW * MT * 16;
}

// Outputs of the splits -> rows of out (pitch ldc), the sink counted once: a block of MW warps per (row, head), each warp adding its
// share of the splits.
constexpr int MW = 4;

template <typename T>
__global__ void __launch_bounds__(MW * 32) merge_kernel(const HyAttend a, const float* __restrict__ o, const float* __restrict__ ml, int splits,
                                                        T* __restrict__ out, int ldc) {
  __shared__ float coef[64];
  __shared__ __align__(16) float part[MW][128];
  const int unit = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = unit / a.heads, h = unit - t * a.heads;
  if (warp == 0) {
    const float* p = ml + static_cast<long long>(unit) * splits * 2;
    const float sink = a.sink ? to_f(static_cast<const T*>(a.sink)[h]) * LOG2E : -FLT_MAX;
    float mv[2], lv[2], m = sink;
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int s = lane + 32 * k;
      mv[k] = s < splits ? p[2 * s] : -FLT_MAX;
      lv[k] = s < splits ? p[2 * s + 1] : 0.f;
      m = fmaxf(m, mv[k]);
    }
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, off));
    float c[2], l = 0.f;
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      c[k] = mv[k] == -FLT_MAX ? 0.f : exp2f(mv[k] - m);
      l += c[k] * lv[k];
    }
    l = warp_sum(l) + (a.sink ? exp2f(sink - m) : 0.f);
    const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
    for (int k = 0; k < 2; ++k) coef[lane + 32 * k] = c[k] * inv;
  }
  const float* src = o + static_cast<long long>(unit) * splits * a.vd;
  T* dst = out + static_cast<long long>(t) * ldc + h * a.vd;
  for (int i0 = 0; i0 < a.vd; i0 += 128) {  // (vd is a multiple of 8)
    const int i = i0 + lane * 4;
    float4 u[4], v = make_float4(0.f, 0.f, 0.f, 0.f);
    const bool live = i < a.vd;
    for (int s0 = warp; s0 < splits; s0 += 4 * MW) {
#pragma unroll
      for (int k = 0; k < 4; ++k)
        u[k] = live && s0 + k * MW < splits ? *reinterpret_cast<const float4*>(src + static_cast<long long>(s0 + k * MW) * a.vd + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      if (s0 == warp) __syncthreads();  // coefficients (first time round) and the partial sums of the columns before
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        const float c = coef[min(s0 + k * MW, 63)];
        v.x += c * u[k].x; v.y += c * u[k].y; v.z += c * u[k].z; v.w += c * u[k].w;
      }
    }
    if (warp >= splits) __syncthreads();
    *reinterpret_cast<float4*>(&part[warp][lane * 4]) = v;
    __syncthreads();
    const int c = threadIdx.x;
    if (i0 + c < a.vd) {
      float r = 0.f;
#pragma unroll
      for (int w = 0; w < MW; ++w) r += part[w][c];
      dst[i0 + c] = from_f<T>(r);
    }
  }
  if (h == a.heads - 1)
    for (int i = a.heads * a.vd + threadIdx.x; i < ldc; i += MW * 32) out[static_cast<long long>(t) * ldc + i] = from_f<T>(0.f);
}

// ------------------------------------------------------------------------------------------------ rows of a range
template <typename T>
__global__ void __launch_bounds__(256) gather_rows_kernel(const HyCache a, const int4* __restrict__ ranges, T* __restrict__ out) {
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

template <typename T>
int attend_t(const HyAttend& a, const float* ql, int qld, const int* positions, const int* row_seq, int n, float* o, void* out, int ldc,
             cudaStream_t s) {
  const size_t smem = sizeof(float) * static_cast<size_t>(a.kd > 4 * a.vd ? a.kd : 4 * a.vd);
  auto go = [&](auto kern) -> int {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    kern<<<dim3(a.heads, n), 128, smem, s>>>(a, ql, qld, positions, row_seq, o, static_cast<T*>(out), ldc);
    return static_cast<int>(cudaGetLastError());
  };
  if (a.vd <= 128) return go(attend_kernel<T, 4>);
  if (a.vd <= 256) return go(attend_kernel<T, 8>);
  if (a.vd <= 512) return go(attend_kernel<T, 16>);
  if (a.vd <= 1024) return go(attend_kernel<T, 32>);
  if (a.vd <= 2048) return go(attend_kernel<T, 64>);
  return static_cast<int>(cudaErrorInvalidValue);
}

template <int MT, int KI, int QI, int NTM>
int decode_t(const HyAttend& a, const bf16* ql, int qld, const int* seq_lens, int B, int splits, float* o, float* ml, cudaStream_t s) {
  const size_t smem = decode_smem(MT, a);
  auto kern = cached_decode_kernel<MT, KI, QI, NTM>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  if (e != cudaSuccess) return static_cast<int>(e);
  const int per = (a.group + MT * 16 - 1) / (MT * 16);
  kern<<<dim3(B, a.heads / a.group * per, splits), DW * 32, smem, s>>>(a, ql, qld, seq_lens, splits, o, ml);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace

int hy_attend(bool f32, const HyAttend& a, const float* q, int qld, const int* positions, const int* row_seq, int T, float* o, void* out,
              int ldc, cudaStream_t s) {
  return f32 ? attend_t<float>(a, q, qld, positions, row_seq, T, o, out, ldc, s) : attend_t<bf16>(a, q, qld, positions, row_seq, T, o, out, ldc, s);
}

bool hy_decode_supported(const HyAttend& a) {
  return a.heads >= 1 && a.group >= 1 && a.kd >= 8 && a.vd >= 8 && (a.kd | a.vd | a.k_col | a.k_step | a.v_col | a.v_step | a.width) % 8 == 0 &&
         key_cols(a) <= 576 && a.vd <= 512 && decode_smem(a.group > 16 ? 2 : 1, a) <= 227 * 1024;
}

int hy_decode(const HyAttend& a, const void* ql, int qld, const int* seq_lens, int B, int splits, float* o, float* ml, cudaStream_t s) {
  if (!hy_decode_supported(a) || qld % 8 != 0 || qld < a.kd || splits < 1 || splits > 64 || a.num_slots > 0x7fffffffll)
    return static_cast<int>(cudaErrorInvalidValue);
  const bf16* q = static_cast<const bf16*>(ql);
  const bool two = a.group > 16;
  if (a.kd <= 128 && a.vd <= 128)
    return two ? decode_t<2, 4, 4, 4>(a, q, qld, seq_lens, B, splits, o, ml, s) : decode_t<1, 4, 4, 2>(a, q, qld, seq_lens, B, splits, o, ml, s);
  if (a.kd <= 256 && a.vd <= 256)
    return two ? decode_t<2, 8, 8, 8>(a, q, qld, seq_lens, B, splits, o, ml, s) : decode_t<1, 8, 8, 4>(a, q, qld, seq_lens, B, splits, o, ml, s);
  return two ? decode_t<2, 18, 10, 16>(a, q, qld, seq_lens, B, splits, o, ml, s) : decode_t<1, 18, 18, 8>(a, q, qld, seq_lens, B, splits, o, ml, s);
}

int hy_decode_merge(bool f32, const HyAttend& a, const float* o, const float* ml, int splits, int B, void* out, int ldc, cudaStream_t s) {
  if (splits < 1 || splits > 64) return static_cast<int>(cudaErrorInvalidValue);
  if (f32) merge_kernel<float><<<B * a.heads, MW * 32, 0, s>>>(a, o, ml, splits, static_cast<float*>(out), ldc);
  else merge_kernel<bf16><<<B * a.heads, MW * 32, 0, s>>>(a, o, ml, splits, static_cast<bf16*>(out), ldc);
  return static_cast<int>(cudaGetLastError());
}

int hy_gather_rows(bool f32, const HyCache& a, const int* ranges, int n, int max_rows, void* out, cudaStream_t s) {
  if (n <= 0 || max_rows <= 0) return 0;
  const dim3 grid((max_rows + 7) / 8, n);
  const int4* rg = reinterpret_cast<const int4*>(ranges);
  if (f32)
    gather_rows_kernel<float><<<grid, 256, 0, s>>>(a, rg, static_cast<float*>(out));
  else
    gather_rows_kernel<bf16><<<grid, 256, 0, s>>>(a, rg, static_cast<bf16*>(out));
  return static_cast<int>(cudaGetLastError());
}

}  // namespace mb
