// Prompt attention over gathered cache rows on tcgen05: causal, with an optional sliding window and an optional sink per head.
//
// Same pipeline as attention_fwd.cu (TMA producer warp, MMA issuer warp, two softmax threads per query row, scores double
// buffered and the output accumulated in TMEM); what differs:
//   * keys and values are column ranges of the rows they come from, wherever these are: a key head's own 64-column boxes, and
//     (SHARED, latent attention) one more box of other rows that all heads have in common. The score product runs over both,
//     queries carry zeros where a box reaches past its part, so that nothing is copied next to anything;
//   * queries see keys in (position - window, position]: a tile starts at the first block its first query sees;
//   * value width and key width differ, and the output goes straight into the rows of the product that follows;
//   * a sink is one more term of the denominator: it enters once, at the end.
#include <cuda.h>
#include <float.h>
#include <stdio.h>

#include <mutex>
#include <string>

#include "hybrid.h"
#include "ptx.cuh"

namespace mb {
namespace {

constexpr int BM = 128;                     // query rows per tile
constexpr int BN = 128;                     // keys per block
constexpr int ATOM = 128 * 128;             // bytes: 128 rows x 64 bf16
constexpr int LP_THREADS = 320;

struct LpArgs {
  const int4* tiles;
  int heads, group, vdim, window;
  int k_col, k_step, v_col, v_step;  // columns of key head g: k_col + g * k_step ..
  int shared_col;                    // of the part all heads share, in its own rows
  const __nv_bfloat16* sink;
  __nv_bfloat16* out;
  int ldc;
  float scale_log2;
  int* status;
};

__device__ __forceinline__ uint32_t swz(int row, int chunk16) { return static_cast<uint32_t>(row * 128 + ((chunk16 ^ (row & 7)) << 4)); }
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int NN, int NV, bool SHARED>
struct Lp {
  static constexpr int KA = NN + (SHARED ? 1 : 0);  // 64-column atoms of a key: NN own, one shared
  static constexpr int VST = KA <= 2 ? 2 : 1;       // value stages (one where keys take the room; its load hides behind the softmax)
  static constexpr int Q_BYTES = KA * ATOM, P_BYTES = 2 * ATOM, K_BYTES = KA * ATOM, V_BYTES = NV * ATOM;
  static constexpr int SMEM = Q_BYTES + P_BYTES + 2 * K_BYTES + VST * V_BYTES + 256 + 1024;
};

template <int NN, int NV, bool SHARED>
__global__ void __launch_bounds__(LP_THREADS, 1)
cached_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_kv,
                      const __grid_constant__ CUtensorMap map_c, const LpArgs p) {
  using L = Lp<NN, NV, SHARED>;
  constexpr int VST = L::VST;
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t q_s = base;
  const uint32_t p_s = q_s + L::Q_BYTES;
  const uint32_t k_s = p_s + L::P_BYTES;
  const uint32_t v_s = k_s + 2 * L::K_BYTES;
  const uint32_t bars = v_s + VST * L::V_BYTES;
  auto BAR = [&](int i) { return bars + 8u * i; };
  constexpr int B_QF = 0, B_KF = 1, B_KE = 3, B_VF = 5, B_VE = 7, B_SF = 9, B_PF = 11, B_PVD = 12, B_PAIR = 13;
  const uint32_t tmem_slot = bars + 8u * 17;
  __shared__ int abort_s;
  __shared__ float xch[2][2][BM];
  __shared__ uint32_t tmem_base_s;
  volatile int* abort_flag = &abort_s;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int4 tile = p.tiles[blockIdx.x];
  const int head = blockIdx.y;
  const int q_row0 = tile.x, q_rows = tile.y, kv_row0 = tile.z, q_pos0 = tile.w;
  const int j0 = p.window > 0 ? max(0, q_pos0 - p.window + 1) / BN : 0;  // first block any query of the tile sees
  const int n_blocks = (q_pos0 + q_rows + BN - 1) / BN - j0;              // (at least one: a query sees itself)

  if (threadIdx.x == 0) {
    abort_s = 0;
    mbar_init(BAR(B_QF), 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(BAR(B_KF + s), 1);
      mbar_init(BAR(B_KE + s), 1);
      mbar_init(BAR(B_VF + s), 1);
      mbar_init(BAR(B_VE + s), 1);
      mbar_init(BAR(B_SF + s), 1);
    }
    mbar_init(BAR(B_PF), 8);
    mbar_init(BAR(B_PVD), 1);
    for (int s = 0; s < 4; ++s) mbar_init(BAR(B_PAIR + s), 2);
    fence_barrier_init();
    prefetch_tensormap(&map_q);
    prefetch_tensormap(&map_kv);
    if (SHARED) prefetch_tensormap(&map_c);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (threadIdx.x == 0) {
    uint32_t v;
    asm volatile("ld.shared.u32 %0, [%1];" : "=r"(v) : "r"(tmem_slot));
    tmem_base_s = v;
  }
  __syncthreads();
  const uint32_t tmem = tmem_base_s;
  auto T_S = [&](int b) { return tmem + static_cast<uint32_t>(b) * 128u; };
  const uint32_t t_O = tmem + 256;
  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      bool ok = true;
      const int g = head / p.group, k_col = p.k_col + g * p.k_step, v_col = p.v_col + g * p.v_step;
      mbar_expect_tx(BAR(B_QF), L::Q_BYTES);
#pragma unroll
      for (int i = 0; i < L::KA; ++i) tma_load_2d(q_s + i * ATOM, &map_q, BAR(B_QF), (head * L::KA + i) * 64, q_row0);
      auto load_k = [&](int j) -> bool {
        const int st = j & 1, row = kv_row0 + (j0 + j) * BN;
        if (!mbar_wait(BAR(B_KE + st), ((j >> 1) & 1) ^ 1, abort_flag, p.status, ERR_WAIT_EMPTY)) return false;
        mbar_expect_tx(BAR(B_KF + st), L::K_BYTES);
        const uint32_t dst = k_s + st * L::K_BYTES;
#pragma unroll
        for (int i = 0; i < NN; ++i) tma_load_2d(dst + i * ATOM, &map_kv, BAR(B_KF + st), k_col + i * 64, row);
        if (SHARED) tma_load_2d(dst + NN * ATOM, &map_c, BAR(B_KF + st), p.shared_col, row);
        return true;
      };
      auto load_v = [&](int j) -> bool {
        const int st = j % VST, row = kv_row0 + (j0 + j) * BN;
        if (!mbar_wait(BAR(B_VE + st), ((j / VST) & 1) ^ 1, abort_flag, p.status, ERR_WAIT_EMPTY)) return false;
        mbar_expect_tx(BAR(B_VF + st), L::V_BYTES);
        const uint32_t dst = v_s + st * L::V_BYTES;
#pragma unroll
        for (int i = 0; i < NV; ++i)
          tma_load_2d(dst + i * ATOM, &map_kv, BAR(B_VF + st), v_col + i * 64, row);
        return true;
      };
      ok = load_k(0);
      for (int j = 0; ok && j < n_blocks; ++j) {
        if (j + 1 < n_blocks) ok = load_k(j + 1);
        if (ok) ok = load_v(j);
      }
      if (!ok) {  // give copies in flight a bounded chance to land before shared memory is released
        const unsigned long long t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 2000000ull) {
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    constexpr uint32_t idesc_qk = make_idesc_bf16(BM, BN, false, false);
    constexpr uint32_t idesc_pv = make_idesc_bf16(BM, NV * 64, false, true);
    bool ok = mbar_wait(BAR(B_QF), 0, abort_flag, p.status, ERR_WAIT_FULL);
    auto issue_qk = [&](int j) -> bool {
      const int st = j & 1;
      if (!mbar_wait(BAR(B_KF + st), (j >> 1) & 1, abort_flag, p.status, ERR_WAIT_FULL)) return false;
      tc_fence_after();
      if (lane == 0) {
        const uint32_t kb = k_s + st * L::K_BYTES;
#pragma unroll
        for (int k = 0; k < L::KA * 4; ++k) {
          const uint32_t off = (k >> 2) * ATOM + (k & 3) * 32;
          umma_f16(T_S(j & 1), make_smem_desc(q_s + off, 16, 1024), make_smem_desc(kb + off, 16, 1024), idesc_qk, k > 0 ? 1u : 0u);
        }
        umma_commit(BAR(B_KE + st));
        umma_commit(BAR(B_SF + (j & 1)));
      }
      __syncwarp();
      return true;
    };
    if (ok) ok = issue_qk(0);
    for (int j = 0; ok && j < n_blocks; ++j) {
      // S[(j+1)&1] was last read for block j-1, whose softmax finished before p_full(j-1) was observed below.
      if (j + 1 < n_blocks) ok = issue_qk(j + 1);
      if (!ok) break;
      const int st = j % VST;
      if (!mbar_wait(BAR(B_PF), j & 1, abort_flag, p.status, ERR_WAIT_TMEM_EMPTY) ||
          !mbar_wait(BAR(B_VF + st), (j / VST) & 1, abort_flag, p.status, ERR_WAIT_FULL)) {
        ok = false;
        break;
      }
      tc_fence_after();
      if (lane == 0) {
        const uint32_t vb = v_s + st * L::V_BYTES;
#pragma unroll
        for (int k = 0; k < BN / 16; ++k) {
          const uint64_t adesc = make_smem_desc(p_s + (k >> 2) * ATOM + (k & 3) * 32, 16, 1024);
          const uint64_t bdesc = make_smem_desc(vb + k * 2048, ATOM, 1024);
          umma_f16(t_O, adesc, bdesc, idesc_pv, (j > 0 || k > 0) ? 1u : 0u);
        }
        umma_commit(BAR(B_VE + st));
        umma_commit(BAR(B_PVD));
      }
      __syncwarp();
    }
  } else {
    // ------------------------------------------------------------------ softmax (warps 2..9)
    const int quad = warp & 3;
    const int half = (warp - 2) >> 2;
    const int row = quad * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t pair_bar = BAR(B_PAIR + quad);
    const int qpos = q_pos0 + row;
    const int first = p.window > 0 ? qpos - p.window + 1 : 0;   // this row sees keys first .. qpos
    constexpr int OC = NV * 32;                                  // output columns of this thread
    float m_used = -INFINITY, l = 0.f;
    uint32_t sr[64];
    bool ok = true;
    for (int j = 0; j < n_blocks; ++j) {
      const int b = j & 1, k0 = (j0 + j) * BN;
      if (!mbar_wait(BAR(B_SF + b), (j >> 1) & 1, abort_flag, p.status, ERR_WAIT_TMEM_FULL)) {
        ok = false;
        break;
      }
      tc_fence_after();
      const uint32_t s_addr = T_S(b) + lane_addr + half * 64;
      tmem_ld_32x32(s_addr, *reinterpret_cast<uint32_t(*)[32]>(&sr[0]));
      tmem_ld_32x32(s_addr + 32, *reinterpret_cast<uint32_t(*)[32]>(&sr[32]));
      tmem_ld_wait();
      float mx = -INFINITY;
      const int col0 = k0 + half * 64;
      // masked where the block reaches past the tile's first query, or before what its last query sees
      if (k0 + BN - 1 > q_pos0 || (p.window > 0 && k0 < q_pos0 + BM - p.window)) {
#pragma unroll
        for (int i = 0; i < 64; ++i) {
          float s = __uint_as_float(sr[i]) * p.scale_log2;
          s = (col0 + i > qpos || col0 + i < first) ? -INFINITY : s;
          sr[i] = __float_as_uint(s);
          mx = fmaxf(mx, s);
        }
      } else {
#pragma unroll
        for (int i = 0; i < 64; ++i) {
          const float s = __uint_as_float(sr[i]) * p.scale_log2;
          sr[i] = __float_as_uint(s);
          mx = fmaxf(mx, s);
        }
      }
      xch[b][half][row] = mx;
      __syncwarp();
      if (lane == 0) mbar_arrive(pair_bar);
      if (!mbar_wait(pair_bar, j & 1, abort_flag, p.status, ERR_WAIT_PEER)) {
        ok = false;
        break;
      }
      mx = fmaxf(mx, xch[b][half ^ 1][row]);
      const float m_new = fmaxf(m_used, mx);
      const bool grow = m_new > m_used + 8.f;  // also true on the first finite maximum
      const bool any_grow = __any_sync(0xffffffffu, grow);
      float alpha = 1.f;
      if (any_grow) {
        alpha = (m_new == -INFINITY) ? 1.f : ex2(m_used - m_new);
        m_used = m_new;
        l *= alpha;
      }
      const float base_m = (m_used == -INFINITY) ? 0.f : m_used;
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        const float p0 = ex2(__uint_as_float(sr[2 * i]) - base_m);
        const float p1 = ex2(__uint_as_float(sr[2 * i + 1]) - base_m);
        sum += p0 + p1;
        sr[i] = pack_bf16(p0, p1);
      }
      l += sum;
      if (j > 0) {
        if (!mbar_wait(BAR(B_PVD), (j - 1) & 1, abort_flag, p.status, ERR_WAIT_TMEM_FULL)) {
          ok = false;
          break;
        }
        tc_fence_after();
        if (any_grow) {
          uint32_t o[32];
#pragma unroll 1
          for (int c = 0; c < OC / 32; ++c) {
            const uint32_t o_addr = t_O + lane_addr + half * OC + c * 32;
            tmem_ld_32x32(o_addr, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st_32x32(o_addr, o);
          }
          tmem_st_wait();
        }
      }
      const uint32_t p_row = p_s + half * ATOM;
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(p_row + swz(row, c)), "r"(sr[4 * c]), "r"(sr[4 * c + 1]),
                     "r"(sr[4 * c + 2]), "r"(sr[4 * c + 3])
                     : "memory");
      }
      fence_proxy_async();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(BAR(B_PF));
    }
    // ---- epilogue: O / l -> bf16
    if (ok && n_blocks > 0) ok = mbar_wait(BAR(B_PVD), (n_blocks - 1) & 1, abort_flag, p.status, ERR_WAIT_TMEM_FULL);
    if (ok) {
      tc_fence_after();
      const int b = n_blocks & 1;
      xch[b][half][row] = l;
      __syncwarp();
      if (lane == 0) mbar_arrive(pair_bar);
      ok = mbar_wait(pair_bar, n_blocks & 1, abort_flag, p.status, ERR_WAIT_PEER);
      if (ok) {
        float l_tot = l + xch[b][half ^ 1][row];
        if (p.sink) l_tot += ex2(__bfloat162float(p.sink[head]) * 1.4426950408889634f - m_used);
        const float inv = l_tot > 0.f ? 1.f / l_tot : 0.f;
        const bool live = row < q_rows;
        __nv_bfloat16* dst = p.out + static_cast<long long>(q_row0 + row) * p.ldc + head * p.vdim + half * OC;
        uint32_t o[32];
#pragma unroll 1
        for (int c = 0; c < OC / 32; ++c) {
          tmem_ld_32x32(t_O + lane_addr + half * OC + c * 32, o);
          tmem_ld_wait();
          if (live) {
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              if (half * OC + c * 32 + i * 8 >= p.vdim) break;
              uint4 v;
              v.x = pack_bf16(__uint_as_float(o[8 * i]) * inv, __uint_as_float(o[8 * i + 1]) * inv);
              v.y = pack_bf16(__uint_as_float(o[8 * i + 2]) * inv, __uint_as_float(o[8 * i + 3]) * inv);
              v.z = pack_bf16(__uint_as_float(o[8 * i + 4]) * inv, __uint_as_float(o[8 * i + 5]) * inv);
              v.w = pack_bf16(__uint_as_float(o[8 * i + 6]) * inv, __uint_as_float(o[8 * i + 7]) * inv);
              *reinterpret_cast<uint4*>(dst + c * 32 + i * 8) = v;
            }
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// ---------------------------------------------------------------------- host side
typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*,
                                  const cuuint64_t*, const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave,
                                  CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
std::string g_lp_err;
EncodeTiledFn g_lp_encode = nullptr;
std::once_flag g_lp_once;

int lp_fail(const std::string& m) {
  g_lp_err = m;
  return -1;
}

// bf16 [rows, cols] with row pitch ld; box = 64 columns x 128 rows, 128-byte swizzle, zeros outside.
int lp_map(CUtensorMap* map, const void* ptr, long long rows, long long cols, long long ld) {
  std::call_once(g_lp_once, [] {
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &q) == cudaSuccess && q == cudaDriverEntryPointSuccess)
      g_lp_encode = reinterpret_cast<EncodeTiledFn>(fn);
  });
  if (!g_lp_encode) return lp_fail("cuTensorMapEncodeTiled is not available");
  if ((reinterpret_cast<uintptr_t>(ptr) & 15) != 0 || (ld * 2) % 16 != 0) return lp_fail("attention operands need 16-byte aligned rows");
  cuuint64_t dims[2] = {static_cast<cuuint64_t>(cols), static_cast<cuuint64_t>(rows)};
  cuuint64_t strides[1] = {static_cast<cuuint64_t>(ld) * 2};
  cuuint32_t box[2] = {64u, 128u};
  cuuint32_t estr[2] = {1u, 1u};
  CUresult r = g_lp_encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), dims, strides, box, estr,
                           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (r != CUDA_SUCCESS) return lp_fail("cuTensorMapEncodeTiled failed with code " + std::to_string(int(r)));
  return 0;
}

template <int NN, int NV, bool SHARED>
int lp_launch(const CUtensorMap& mq, const CUtensorMap& mkv, const CUtensorMap& mc, const LpArgs& a, int n_tiles, cudaStream_t s) {
  auto kern = cached_prefill_kernel<NN, NV, SHARED>;
  constexpr int smem = Lp<NN, NV, SHARED>::SMEM;
  static_assert(smem <= 227 * 1024, "shared memory of the prompt attention kernel");
  if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
    return lp_fail("cudaFuncSetAttribute(MaxDynamicSharedMemorySize) failed for prompt attention");
  kern<<<dim3(n_tiles, a.heads), LP_THREADS, smem, s>>>(mq, mkv, mc, a);
  if (cudaGetLastError() != cudaSuccess) return lp_fail("prompt attention launch failed");
  return 0;
}

template <bool SHARED>
int lp_pick(int q_pad, const CUtensorMap& mq, const CUtensorMap& mkv, const CUtensorMap& mc, const LpArgs& p, int n_tiles, cudaStream_t s) {
  if (q_pad == 64) return p.vdim <= 64 ? lp_launch<1, 1, SHARED>(mq, mkv, mc, p, n_tiles, s) : lp_launch<1, 2, SHARED>(mq, mkv, mc, p, n_tiles, s);
  return p.vdim <= 64 ? lp_launch<2, 1, SHARED>(mq, mkv, mc, p, n_tiles, s) : lp_launch<2, 2, SHARED>(mq, mkv, mc, p, n_tiles, s);
}

}  // namespace

const char* hy_prefill_last_error() { return g_lp_err.c_str(); }

bool hy_prefill_supported(int dim, int rot, int vdim, int rank, int width) {
  // every box starts at a column that is a multiple of 8 (16 bytes)
  return dim % 8 == 0 && vdim % 8 == 0 && rot % 8 == 0 && rank % 8 == 0 && width % 8 == 0 && dim >= 8 && dim <= 128 && rot >= 0 &&
         rot <= 64 && vdim >= 8 && vdim <= 128;
}

int hy_prefill(const HyPrefill& a, const int* tiles, int n_tiles, int T, void* out, int ldc, cudaStream_t s) {
  const bool shared = a.shared != nullptr;
  if (!hy_prefill_supported(a.dim, shared ? a.rot : 0, a.vdim, a.shared_col, shared ? a.shared_width : 0) ||
      (a.k_col | a.k_step | a.v_col | a.v_step) % 8 != 0 || (shared && a.rot < 8))
    return lp_fail("head sizes are not supported by the tensor-core prompt attention");
  if ((a.q_pad != 64 && a.q_pad != 128) || a.q_pad < a.dim) return lp_fail("queries must be padded to 64 or 128 columns");
  if (ldc % 8 != 0 || (reinterpret_cast<uintptr_t>(out) & 15) != 0) return lp_fail("the output rows must be 16-byte aligned");
  if (n_tiles == 0) return 0;
  CUtensorMap mq, mkv, mc;
  const long long qw = static_cast<long long>(a.heads) * (a.q_pad + (shared ? 64 : 0));
  if (lp_map(&mq, a.q, T, qw, qw)) return -1;
  if (lp_map(&mkv, a.kv, a.ctx_rows, a.kv_cols, a.kv_ld)) return -1;
  mc = mkv;
  if (shared && lp_map(&mc, a.shared, a.ctx_rows, a.shared_width, a.shared_width)) return -1;
  LpArgs p;
  p.tiles = reinterpret_cast<const int4*>(tiles);
  p.heads = a.heads;
  p.group = a.group;
  p.vdim = a.vdim;
  p.window = a.window;
  p.k_col = a.k_col; p.k_step = a.k_step; p.v_col = a.v_col; p.v_step = a.v_step;
  p.shared_col = a.shared_col;
  p.sink = static_cast<const __nv_bfloat16*>(a.sink);
  p.out = static_cast<__nv_bfloat16*>(out);
  p.ldc = ldc;
  p.scale_log2 = a.scale * 1.4426950408889634f;
  p.status = a.status;
  return shared ? lp_pick<true>(a.q_pad, mq, mkv, mc, p, n_tiles, s) : lp_pick<false>(a.q_pad, mq, mkv, mc, p, n_tiles, s);
}

}  // namespace mb
