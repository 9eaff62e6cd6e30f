// Host API of the kernels behind models with a layer plan (mixers that differ from layer to layer). `f32` selects the
// 32-bit instantiation: activations and weights are then float, otherwise bf16. The residual stream, recurrent state,
// norms, angles and attention scores are fp32 in both.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace mb {

// ---- hybrid_ops.cu
// x[t] = table[token]; h[t] = dynamic-tanh norm of it.
int hy_embed_norm(bool f32, const int* tokens, int T, const void* table, int V, int H, const void* w, const void* b,
                  const void* alpha, float* x, void* h, int* status, cudaStream_t s);

// Gated feed-forward and column padding of a fused output row: cat[t] = [mixer (written elsewhere) | 0 | silu(gate) * up | 0].
struct HyCat {
  const void* proj;      // fused input products [T, ld]
  long long ld;
  int gate, up, ff;      // column starts of gate and up rows, width (0 = no feed-forward)
  void* cat;             // [T, ldc]
  int ldc, mixed, down;  // columns the mixer fills, first column of the feed-forward's part
};

// Mamba-2 tail: cat[t, :inner] = group-wise RMS norm of (y * silu(z)) * w, and the feed-forward part of the row.
int hy_mamba_tail(bool f32, const void* y, const void* w, int inner, int norm_groups, float eps, const HyCat& c, int T,
                  cudaStream_t s);

// Latent-attention head of a layer: cq = RMS norm of the query latent; the key / value latent (RMS normed) and the rotated
// key part go to their cache row; the feed-forward part of the row.
struct HyLatentIn {
  int dq, q_rank;        // columns of proj
  int dkv;               // first column of the own latent, -1: the layer reads another layer's rows
  int kv_rank, rot_dim;
  const void *q_norm, *kv_norm;
  const float* freq;     // [rot_dim / 2]
  const int *positions, *slots;
  void* cq;              // [T, q_rank]
  void* rows;            // cache [num_slots, width]
  int width;
  long long num_slots;
  float eps;
  int* status;
};
int hy_latent_in(bool f32, const HyLatentIn& a, const HyCat& c, int T, cudaStream_t s);

// Per-layer token input, residual and next norm, one kernel (clusters of 8 CTAs): x' = x + delta (delta may be null),
// g = gelu(gate x') * e, y = proj g, x = x' + rmsnorm(y) * norm, h = dynamic-tanh(x).
struct HySide {
  float* x;              // [T, H], updated
  const float* delta;
  const int* tokens;
  const void *gate, *proj, *norm, *embed;  // [sd, H], [H, sd], [H], [V, embed_ld] (columns embed_col ..)
  int sd, H, V, embed_ld, embed_col;
  const void *nw, *nb, *na;                // next norm
  void* h;
  float eps;
  int* status;
};
int hy_side_fused(bool f32, const HySide& a, int T, cudaStream_t s);
// The same in pieces around tensor-core products, for many rows: x += delta (may be null) and its bf16 copy, then g from the gate
// product, then the rest.
int hy_cast_rows(float* x, const float* delta, void* out_bf16, long long n, cudaStream_t s);
int hy_side_gate(bool f32, const float* z, const HySide& a, void* g, int T, cudaStream_t s);
int hy_side_finish(bool f32, const float* y, const HySide& a, int T, cudaStream_t s);

// ---- mamba2.cu
struct HyMamba {
  const void* proj;      // [T, ld], columns [z | x | B | C | dt] from column 0
  long long ld;
  long long xld;         // rows the recurrence itself reads (xbc): pitch, first columns of x, B and C
  int x_col, b_col, c_col;
  const float* log2_decay;  // [heads] or null: a constant decay per token instead of exp(-exp(A_log) dt), and dt = 1
  int heads, P, N, groups, taps;
  const void *conv_w, *conv_b, *dt_bias, *A_log, *D;
  void* ring;            // [sequences, taps, channels]: input of position p in row p % taps
  float* state;          // [sequences, heads, P, N]
  int sequences;
  const int *cu, *ctx, *slots;  // prefill: row offsets, cached tokens, state row of every sequence
  int nseq;
  int* status;
};
// Prefill: convolution + silu of all rows into xbc [T, channels]; `tiles` int32 [n][4] = {sequence, first row, rows, 0}.
int hy_conv(bool f32, const HyMamba& a, const int* tiles, int n_tiles, void* xbc, cudaStream_t s);
// Sequential scan (any sizes, exact fp32): y [T, heads * P]
int hy_scan(bool f32, const HyMamba& a, const void* xbc, void* y, cudaStream_t s);
// Chunked scan on the tensor cores (bf16). `chunks` int32 [n][4] = {sequence, first row, rows, chunk index in sequence},
// sequence by sequence; `first_chunk` [nseq + 1]; work: fp32 [n, heads, P, N], decay: fp32 [n, heads], before: bf16
// [n, heads, 2, P, N].
bool hy_chunk_scan_supported(int P, int N, int heads, int groups);
constexpr int HY_CHUNK = 128;
// The scan over chunks on its own: decay [n, heads], or with `cols` [n, heads, 2, N]: one per column, and a factor for `before`.
int hy_chunk_pass(const HyMamba& a, const int* first_chunk, const float* decay, bool cols, const float* work, void* before, cudaStream_t s);
int hy_chunk_scan(const HyMamba& a, const void* xbc, const int* chunks, int n_chunks, const int* first_chunk, float* work,
                  float* decay, void* before, void* y, cudaStream_t s);
// One token per sequence: convolution, state update and output in one kernel. positions[b] = 0 starts from a zero state.
int hy_mamba_step(bool f32, const HyMamba& a, const int* positions, int B, void* y, cudaStream_t s);

// ---- cached_attention.cu
struct HyCache {
  const void* rows;      // cache [num_slots, width]
  long long num_slots;
  int width;
  const int* table;      // [B, max_pages]
  int max_pages, page_size;
  int* status;
};
// Query head h reads key head h / group: its key is columns k_col + (h / group) * k_step .. + kd of a row, its value v_col + .. + vd.
struct HyAttend : HyCache {
  int heads, group, kd, vd;
  int k_col, k_step, v_col, v_step;
  int window;            // 0: all earlier tokens
  float scale;
  const void* sink;      // [heads] or null
};
// Any sizes, any number of rows: row t is position positions[t] of sequence row_seq[t] (null: sequence t). q [T, heads, qld] fp32;
// the result goes to o [T, heads, vd] fp32, or (o null) to rows of out, pitch ldc.
int hy_attend(bool f32, const HyAttend& a, const float* q, int qld, const int* positions, const int* row_seq, int T, float* o, void* out,
              int ldc, cudaStream_t s);
// Decode on the tensor cores (bf16, one row per sequence): partial outputs of each split, fp32 o [B, heads, splits, vd],
// ml [B, heads, splits, 2] (maximum and sum, base 2). q [B, heads, qld] bf16.
bool hy_decode_supported(const HyAttend& a);
int hy_decode(const HyAttend& a, const void* q, int qld, const int* seq_lens, int B, int splits, float* o, float* ml, cudaStream_t s);
int hy_decode_merge(bool f32, const HyAttend& a, const float* o, const float* ml, int splits, int B, void* out, int ldc, cudaStream_t s);
// Cached rows of `n` ranges {sequence, first position, first output row, rows} into out [.., width].
int hy_gather_rows(bool f32, const HyCache& a, const int* ranges, int n, int max_rows, void* out, cudaStream_t s);

// ---- cached_prefill.cu (tcgen05): prompt attention over gathered rows.
struct HyPrefill {
  const void* q;         // [T, heads, q_pad (+ 64 with a shared part)], zeros past dim (and past rot)
  int heads, group, dim, vdim, q_pad, window;
  float scale;
  const void* kv;        // [ctx_rows, kv_ld], kv_cols columns; columns of a key head as in HyAttend
  long long ctx_rows, kv_cols, kv_ld;
  int k_col, k_step, v_col, v_step;
  const void* shared;    // [ctx_rows, shared_width] or null: a key part of rot columns from shared_col that all heads have in common
  int rot, shared_col, shared_width;
  const void* sink;      // [heads] bf16 or null
  int* status;
};
// tiles int32 [n][4] {q row, q rows, first key row, position of the first query relative to the first key row}; out [T, ldc], head h
// at column h * vdim.
bool hy_prefill_supported(int dim, int rot, int vdim, int rank, int width);
int hy_prefill(const HyPrefill& a, const int* tiles, int n_tiles, int T, void* out, int ldc, cudaStream_t s);
const char* hy_prefill_last_error();

// ---- latent_attention.cu
struct HyLatent : HyCache {
  int heads, dim, rot, vdim, rank, window;
  float scale;
  const void* ukv;       // [heads * dim | heads * vdim rows, rank]
  const float* freq;
};
// The cache as its absorbed form reads it: one key head, keys [rank + rot], values the first rank columns.
HyAttend hy_latent_view(const HyLatent& a);
// Queries into latent space: ql[t, h] = W_uk[h]^T q_nope (rank values) | rotated part | zeros up to qld. ql [T, heads, qld] is
// fp32 (the plain kernel reads it) or bf16 (the tensor-core decode kernel).
int hy_absorb_q(bool f32, const HyLatent& a, const void* q, const int* positions, int T, void* ql, int qld, bool out_f32,
                cudaStream_t s);
// Output heads from latent outputs: cat[t, h * vdim + v] = W_uv[h] o[t, h]; `splits` > 1 merges partial results first.
int hy_latent_up(bool f32, const HyLatent& a, const float* o, const float* ml, int splits, int T, void* cat, int ldc,
                 cudaStream_t s);
// Rotated queries in the padded per-head layout of the prefill kernel: [T, heads, nope_pad + rot_pad], zeros in the pads.
int hy_pad_q(const HyLatent& a, const void* q, const int* positions, int T, int nope_pad, int rot_pad, void* out, cudaStream_t s);

// ---- linear_attention.cu: S <- S diag(decay) + v k^T, o = S q, on the per-sequence state [heads, P, N] fp32
struct HyLinear {
  const void* proj;      // [T, ld]: columns of values, keys, queries, output gates and (rank > 0) the decay's low-rank input
  long long ld;
  int v, k, q, g, u;
  int heads, P, N;
  float q_scale, k_scale;
  const float* freq;     // rotation of queries and keys in halves of the first `rot` dimensions
  int rot;
  const float* decay_m1; // [heads]: decay - 1 (rank = 0)
  const float* log2_decay;
  int rank;
  const void *a2, *a2_bias;  // [heads * N, rank], [heads * N]: decay = sigmoid(a2 u + bias)^(1 / tau)
  float inv_tau;
  const void* norm;      // [P] or null: weight of the output norm
  float eps;
  float* state;          // [sequences, heads, P, N]
  int sequences;
  const int *cu, *ctx, *slots;
  int nseq;
  int* status;
};
// Decay of every row and channel: out [T, heads * N] = decay - 1, or with chunk tables (int32 [n][4] as in hy_chunk_scan) the running
// sum of log2(decay) over each chunk.
int hy_linear_gate(bool f32, const HyLinear& a, const int* chunks, int n_chunks, int T, float* out, cudaStream_t s);
// Sequential scan (any sizes, fp32): keys and queries already rotated and scaled by hy_head_rows; decays from `gate` (rank > 0).
int hy_linear_scan(bool f32, const HyLinear& a, const float* gate, void* y, cudaStream_t s);
// Chunked scan on the tensor cores (bf16) with a decay per channel; gate holds the running sums. work fp32 [n, heads, P, N], decay fp32
// [n, heads, 2, N], wide int32 [n, heads], before bf16 [n, heads, 2, P, N].
bool hy_linear_chunks_supported(int P, int N);
int hy_linear_chunks(const HyLinear& a, const float* gate, const int* chunks, int n_chunks, const int* first_chunk, float* work, float* decay,
                     int* wide, void* before, void* y, cudaStream_t s);
// out[t, h * P ..] = unit-rms(y) (* norm) * silu(g); zeros from heads * P to ldc.
int hy_linear_tail(bool f32, const HyLinear& a, const void* y, int T, void* out, int ldc, cudaStream_t s);
// One token per sequence: rotation, decay, state update, output norm and gate in one kernel. positions[b] = 0 starts from a zero state.
int hy_linear_step(bool f32, const HyLinear& a, const int* positions, int B, void* out, int ldc, cudaStream_t s);

// ---- sequential_ops.cu
// Up to three head-wise operations on projected rows: rotate the first `rot` dimensions in halves, divide by the root mean square,
// scale, and store (in place, to another row layout with padding, or to a cache row).
struct HyHeadOp {
  int src, heads, dim, rot;
  const float* freq;
  bool unit;
  float scale;
  void* dst;             // row t (or, by_slot, row slots[t]), pitch ld, head h at column col + h * pitch; zeros up to the pitch
  long long ld;
  int col, pitch;
  int tail;              // zero columns after the last head
  bool by_slot, f32;     // f32: dst holds fp32
};
struct HyHeadRows {
  HyHeadOp op[3];
  int n;
  const void* proj;
  long long ld;
  const int *positions, *slots;
  long long num_slots;
  float eps;
  int* status;
  float2* turns[3];      // work for many rows: [T, rot / 2] (cosine, sine) per operation, written where `fill` says so; or null
  bool fill[3];
};
int hy_head_rows(bool f32, const HyHeadRows& a, int T, cudaStream_t s);
// out[t] = act(gate) * up, zeros up to ldo. act: 0 silu, 1 relu
int hy_gated_act(bool f32, const void* proj, long long ld, int gate, int up, int ff, int act, int T, void* out, int ldo, cudaStream_t s);
// Around a sublayer's output y: x += layernorm(y) * post, h = layernorm(x) * next. With y2: y = (rms(y) * w1 + rms(y2) * w2) / 2 first.
// With tokens: x = table[token] instead (and no y).
struct HySandwich {
  float* x;              // [T, H]
  const int* tokens;
  const void* table;
  int V;
  const float *y, *y2;
  const void *w1, *w2, *post, *next;
  void* h;
  int H;
  float eps;
  int* status;
};
int hy_sandwich(bool f32, const HySandwich& a, int T, cudaStream_t s);

}  // namespace mb
