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
int hy_chunk_scan(const HyMamba& a, const void* xbc, const int* chunks, int n_chunks, const int* first_chunk, float* work,
                  float* decay, void* before, void* y, cudaStream_t s);
// One token per sequence: convolution, state update and output in one kernel. positions[b] = 0 starts from a zero state.
int hy_mamba_step(bool f32, const HyMamba& a, const int* positions, int B, void* y, cudaStream_t s);

// ---- latent_attention.cu
struct HyLatent {
  int heads, dim, rot, vdim, rank, width, window;
  float scale;
  const void* ukv;       // [heads * dim | heads * vdim rows, rank]
  const float* freq;
  const void* rows;      // cache [num_slots, width]
  long long num_slots;
  const int* table;      // [B, max_pages]
  int max_pages, page_size;
  int* status;
};
// Queries into latent space: ql[t, h] = W_uk[h]^T q_nope (rank values) | rotated part | zeros up to qld. ql [T, heads, qld] is
// fp32 (the plain kernel reads it) or bf16 (the tensor-core decode kernel).
int hy_absorb_q(bool f32, const HyLatent& a, const void* q, const int* positions, int T, void* ql, int qld, bool out_f32,
                cudaStream_t s);
// Any sizes, any number of rows: row t is position positions[t] of sequence row_seq[t] (null: sequence t). o [T, heads, rank].
int hy_latent_attend(bool f32, const HyLatent& a, const void* ql, int qld, const int* positions, const int* row_seq, int T,
                     float* o, cudaStream_t s);
// Output heads from latent outputs: cat[t, h * vdim + v] = W_uv[h] o[t, h]; `splits` > 1 merges partial results first.
int hy_latent_up(bool f32, const HyLatent& a, const float* o, const float* ml, int splits, int T, void* cat, int ldc,
                 cudaStream_t s);
// Decode on the tensor cores (bf16, one row per sequence, rank a multiple of 8 up to 512): partial outputs of each split, fp32
// o [T, heads, splits, rank], ml [T, heads, splits, 2].
bool hy_latent_decode_supported(int heads, int rank, int rot, int width);
int hy_latent_decode(const HyLatent& a, const void* ql, int qld, const int* seq_lens, int B, int splits, float* o, float* ml,
                     cudaStream_t s);
// Cached rows of `n` ranges {sequence, first position, first output row, rows} into out [.., width].
int hy_gather_rows(bool f32, const HyLatent& a, const int* ranges, int n, int max_rows, void* out, cudaStream_t s);
// Rotated queries in the padded per-head layout of the prefill kernel: [T, heads, nope_pad + rot_pad], zeros in the pads.
int hy_pad_q(const HyLatent& a, const void* q, const int* positions, int T, int nope_pad, int rot_pad, void* out, cudaStream_t s);

// ---- latent_prefill.cu (tcgen05): attention over materialised keys / values.
// q [T, heads, nope_pad + 64]; kv [ctx, kv_ld] = per-head keys (dim wide) then per-head values (vdim wide); latent rows
// [ctx, width] give the shared rotated part from column rank. tiles int32 [n][4] {q row, q rows, first key row, position of
// the first query relative to the first key row}. out: cat [T, ldc], head h at column h * vdim.
bool hy_prefill_supported(int dim, int rot, int vdim, int rank, int width);
int hy_latent_prefill(const HyLatent& a, const void* q, int nope_pad, const void* kv, long long kv_ld, const void* latent,
                      long long ctx_rows, const int* tiles, int n_tiles, int T, void* out, int ldc, cudaStream_t s);
const char* hy_prefill_last_error();

}  // namespace mb
