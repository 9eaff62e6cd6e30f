// The `_hybrid` extension: bindings of the planned-layer kernels, with the serving kernels they share with other models.
#include "binding_helpers.h"
#include "hybrid.h"

void register_serving(pybind11::module_& m);  // serve_bindings.cpp

namespace {

using namespace mb_bind;
typedef c10::optional<at::Tensor> OptT;

#define RUN(expr)                                                                              \
  do {                                                                                         \
    const int rc_ = (expr);                                                                    \
    TORCH_CHECK(rc_ == 0, #expr " failed: ", cudaGetErrorString(static_cast<cudaError_t>(rc_))); \
  } while (0)

// The absorbed form with whole 16-byte pieces (queries and rows carry zeros up to there).
mb::HyAttend latent_decode_view(const mb::HyLatent& a) {
  mb::HyAttend v = mb::hy_latent_view(a);
  v.kd = (v.kd + 7) / 8 * 8;
  return v;
}
bool latent_decode_supported(int64_t heads, int64_t rank, int64_t rot, int64_t width) {
  mb::HyLatent a = {};
  a.heads = heads; a.rank = rank; a.rot = rot; a.width = width;
  return mb::hy_decode_supported(latent_decode_view(a));
}

bool is_f32(const at::Tensor& t) {
  TORCH_CHECK(t.is_cuda() && (t.scalar_type() == at::kFloat || t.scalar_type() == at::kBFloat16), "expected a bf16 or fp32 CUDA tensor");
  return t.scalar_type() == at::kFloat;
}
void same(const at::Tensor& t, bool f32, const char* what) {
  TORCH_CHECK(t.is_cuda() && t.is_contiguous() && t.scalar_type() == (f32 ? at::kFloat : at::kBFloat16), what, ": wrong type or layout");
}
#define SAME(t, f) same(t, f, #t)

void embed_norm(const at::Tensor& tokens, const at::Tensor& table, const at::Tensor& w, const at::Tensor& b, const at::Tensor& alpha,
                at::Tensor& x, at::Tensor& h, at::Tensor& status) {
  CHECK_I32(tokens); CHECK_F32(x); CHECK_I32(status);
  const bool f = is_f32(table);
  SAME(table, f); SAME(w, f); SAME(b, f); SAME(alpha, f); SAME(h, f);
  const int64_t T = tokens.numel(), H = table.size(1);
  TORCH_CHECK(w.numel() == H && b.numel() == H && alpha.numel() == 1 && x.numel() == T * H && h.numel() == T * H, "embed_norm: shapes");
  const c10::cuda::CUDAGuard guard(table.device());
  RUN(mb::hy_embed_norm(f, tokens.data_ptr<int>(), T, table.data_ptr(), table.size(0), H, w.data_ptr(), b.data_ptr(), alpha.data_ptr(),
                        x.data_ptr<float>(), h.data_ptr(), status.data_ptr<int>(), cur_stream()));
}

mb::HyCat make_cat(const at::Tensor& proj, at::Tensor& cat, int64_t gate, int64_t up, int64_t ff, int64_t mixed, int64_t down) {
  const bool f = is_f32(proj);
  SAME(proj, f); SAME(cat, f);
  TORCH_CHECK(proj.dim() == 2 && cat.dim() == 2 && proj.size(0) == cat.size(0), "fused rows: shapes");
  TORCH_CHECK(ff == 0 || (gate + ff <= proj.size(1) && up + ff <= proj.size(1) && down + ff <= cat.size(1)), "fused rows: columns");
  TORCH_CHECK(mixed <= cat.size(1), "fused rows: columns");
  mb::HyCat c;
  c.proj = proj.data_ptr(); c.ld = proj.size(1);
  c.gate = gate; c.up = up; c.ff = ff;
  c.cat = cat.data_ptr(); c.ldc = cat.size(1);
  c.mixed = mixed; c.down = down;
  return c;
}

void mamba_tail(const at::Tensor& y, const at::Tensor& w, int64_t norm_groups, double eps, const at::Tensor& proj, at::Tensor& cat,
                int64_t gate, int64_t up, int64_t ff, int64_t down) {
  const bool f = is_f32(y);
  SAME(y, f); SAME(w, f); SAME(proj, f);
  const int64_t inner = w.numel(), T = proj.size(0);
  TORCH_CHECK(y.numel() == T * inner && inner % norm_groups == 0 && proj.size(1) >= inner && cat.size(1) >= inner, "mamba_tail: shapes");
  const mb::HyCat c = make_cat(proj, cat, gate, up, ff, inner, down);
  const c10::cuda::CUDAGuard guard(y.device());
  RUN(mb::hy_mamba_tail(f, y.data_ptr(), w.data_ptr(), inner, norm_groups, eps, c, T, cur_stream()));
}

void latent_in(const at::Tensor& proj, at::Tensor& cat, int64_t gate, int64_t up, int64_t ff, int64_t mixed, int64_t down, int64_t dq,
               const at::Tensor& q_norm, int64_t dkv, int64_t rot_dim, const OptT& kv_norm, const at::Tensor& freq,
               const at::Tensor& positions, const OptT& slots, at::Tensor& cq, const OptT& rows, double eps, at::Tensor& status) {
  const bool f = is_f32(proj);
  const mb::HyCat c = make_cat(proj, cat, gate, up, ff, mixed, down);
  SAME(q_norm, f); SAME(cq, f); CHECK_F32(freq); CHECK_I32(positions); CHECK_I32(status);
  const int64_t T = proj.size(0), qr = q_norm.numel();
  TORCH_CHECK(cq.numel() == T * qr && dq + qr <= proj.size(1) && positions.numel() == T, "latent_in: shapes");
  mb::HyLatentIn a = {};
  a.dq = dq; a.q_rank = qr; a.dkv = dkv; a.rot_dim = rot_dim;
  a.q_norm = q_norm.data_ptr(); a.freq = freq.data_ptr<float>(); a.positions = positions.data_ptr<int>();
  a.cq = cq.data_ptr(); a.eps = eps; a.status = status.data_ptr<int>();
  if (dkv >= 0) {
    TORCH_CHECK(kv_norm.has_value() && slots.has_value() && rows.has_value(), "latent_in: an own latent needs its norm and cache");
    SAME((*kv_norm), f); SAME((*rows), f); CHECK_I32((*slots));
    a.kv_rank = kv_norm->numel(); a.kv_norm = kv_norm->data_ptr(); a.slots = slots->data_ptr<int>();
    a.rows = rows->data_ptr(); a.width = rows->size(1); a.num_slots = rows->size(0);
    TORCH_CHECK(slots->numel() == T && a.width >= a.kv_rank + rot_dim && dkv + a.kv_rank + rot_dim <= proj.size(1) &&
                freq.numel() == rot_dim / 2, "latent_in: shapes");
  }
  const c10::cuda::CUDAGuard guard(proj.device());
  RUN(mb::hy_latent_in(f, a, c, T, cur_stream()));
}

mb::HySide make_side(at::Tensor& x, const OptT& delta, const at::Tensor& tokens, const at::Tensor& gate, const at::Tensor& proj,
                     const at::Tensor& norm, const at::Tensor& embed, int64_t layer, const at::Tensor& nw, const at::Tensor& nb,
                     const at::Tensor& na, at::Tensor& h, double eps, at::Tensor& status) {
  const bool f = is_f32(gate);
  CHECK_F32(x); CHECK_I32(tokens); CHECK_I32(status);
  SAME(gate, f); SAME(proj, f); SAME(norm, f); SAME(embed, f); SAME(nw, f); SAME(nb, f); SAME(na, f); SAME(h, f);
  const int64_t T = x.size(0), H = x.size(1), sd = gate.size(0);
  TORCH_CHECK(gate.size(1) == H && proj.size(0) == H && proj.size(1) == sd && norm.numel() == H && nw.numel() == H && nb.numel() == H &&
              na.numel() == 1 && h.numel() == T * H && tokens.numel() == T && (layer + 1) * sd <= embed.size(1), "token input: shapes");
  mb::HySide a = {};
  a.x = x.data_ptr<float>();
  if (delta.has_value()) {
    CHECK_F32((*delta));
    TORCH_CHECK(delta->numel() == T * H, "token input: delta");
    a.delta = delta->data_ptr<float>();
  }
  a.tokens = tokens.data_ptr<int>();
  a.gate = gate.data_ptr(); a.proj = proj.data_ptr(); a.norm = norm.data_ptr(); a.embed = embed.data_ptr();
  a.sd = sd; a.H = H; a.V = embed.size(0); a.embed_ld = embed.size(1); a.embed_col = layer * sd;
  a.nw = nw.data_ptr(); a.nb = nb.data_ptr(); a.na = na.data_ptr();
  a.h = h.data_ptr(); a.eps = eps; a.status = status.data_ptr<int>();
  return a;
}

#define SIDE_ARGS at::Tensor &x, const OptT &delta, const at::Tensor &tokens, const at::Tensor &gate, const at::Tensor &proj, \
                  const at::Tensor &norm, const at::Tensor &embed, int64_t layer, const at::Tensor &nw, const at::Tensor &nb, \
                  const at::Tensor &na, at::Tensor &h, double eps, at::Tensor &status
#define SIDE_PASS x, delta, tokens, gate, proj, norm, embed, layer, nw, nb, na, h, eps, status

void side_fused(SIDE_ARGS) {
  const mb::HySide a = make_side(SIDE_PASS);
  const c10::cuda::CUDAGuard guard(x.device());
  RUN(mb::hy_side_fused(is_f32(gate), a, x.size(0), cur_stream()));
}
void side_gate(SIDE_ARGS, const at::Tensor& z, at::Tensor& g) {
  const mb::HySide a = make_side(SIDE_PASS);
  CHECK_F32(z); SAME(g, is_f32(gate));
  TORCH_CHECK(z.numel() == x.size(0) * gate.size(0) && g.numel() == z.numel(), "side_gate: shapes");
  const c10::cuda::CUDAGuard guard(x.device());
  RUN(mb::hy_side_gate(is_f32(gate), z.data_ptr<float>(), a, g.data_ptr(), x.size(0), cur_stream()));
}
void side_finish(SIDE_ARGS, const at::Tensor& y) {
  const mb::HySide a = make_side(SIDE_PASS);
  CHECK_F32(y);
  TORCH_CHECK(y.numel() == x.numel(), "side_finish: shapes");
  const c10::cuda::CUDAGuard guard(x.device());
  RUN(mb::hy_side_finish(is_f32(gate), y.data_ptr<float>(), a, x.size(0), cur_stream()));
}
void cast_rows(at::Tensor& x, const OptT& delta, at::Tensor& out) {
  CHECK_F32(x); CHECK_BF16(out);
  TORCH_CHECK(x.numel() == out.numel(), "cast_rows: shapes");
  if (delta.has_value()) { CHECK_F32((*delta)); TORCH_CHECK(delta->numel() == x.numel(), "cast_rows: delta"); }
  const c10::cuda::CUDAGuard guard(x.device());
  RUN(mb::hy_cast_rows(x.data_ptr<float>(), opt_ptr<float>(delta), out.data_ptr(), x.numel(), cur_stream()));
}

// ------------------------------------------------------------------------------------------------ Mamba-2
mb::HyMamba make_mamba(const at::Tensor& proj, int64_t heads, int64_t P, int64_t N, int64_t groups, const at::Tensor& conv_w,
                       const at::Tensor& conv_b, const at::Tensor& dt_bias, const at::Tensor& A_log, const at::Tensor& D, at::Tensor& ring,
                       at::Tensor& state, const at::Tensor& slots, at::Tensor& status) {
  const bool f = is_f32(proj);
  SAME(proj, f); SAME(conv_w, f); SAME(conv_b, f); SAME(dt_bias, f); SAME(A_log, f); SAME(D, f); SAME(ring, f);
  CHECK_F32(state); CHECK_I32(slots); CHECK_I32(status);
  const int64_t inner = heads * P, ch = inner + 2 * groups * N;
  TORCH_CHECK(heads > 0 && groups > 0 && heads % groups == 0 && proj.dim() == 2 && proj.size(1) >= inner + ch + heads, "mamba: projection columns");
  TORCH_CHECK(conv_w.size(0) == ch && conv_b.numel() == ch && dt_bias.numel() == heads && A_log.numel() == heads && D.numel() == heads, "mamba: weights");
  TORCH_CHECK(ring.dim() == 3 && ring.size(1) == conv_w.size(1) && ring.size(2) == ch, "mamba: convolution state");
  TORCH_CHECK(state.dim() == 4 && state.size(0) == ring.size(0) && state.size(1) == heads && state.size(2) == P && state.size(3) == N, "mamba: state");
  mb::HyMamba a = {};
  a.proj = proj.data_ptr(); a.ld = proj.size(1);
  a.heads = heads; a.P = P; a.N = N; a.groups = groups; a.taps = conv_w.size(1);
  a.conv_w = conv_w.data_ptr(); a.conv_b = conv_b.data_ptr(); a.dt_bias = dt_bias.data_ptr(); a.A_log = A_log.data_ptr(); a.D = D.data_ptr();
  a.ring = ring.data_ptr(); a.state = state.data_ptr<float>(); a.sequences = state.size(0);
  a.slots = slots.data_ptr<int>(); a.status = status.data_ptr<int>();
  a.xld = ch; a.x_col = 0; a.b_col = inner; a.c_col = inner + groups * N;
  return a;
}
#define MAMBA_ARGS const at::Tensor &proj, int64_t heads, int64_t P, int64_t N, int64_t groups, const at::Tensor &conv_w, const at::Tensor &conv_b, \
                   const at::Tensor &dt_bias, const at::Tensor &A_log, const at::Tensor &D, at::Tensor &ring, at::Tensor &state,   \
                   const at::Tensor &slots, at::Tensor &status
#define MAMBA_PASS proj, heads, P, N, groups, conv_w, conv_b, dt_bias, A_log, D, ring, state, slots, status

void mamba_step(MAMBA_ARGS, const at::Tensor& positions, at::Tensor& y) {
  const mb::HyMamba a = make_mamba(MAMBA_PASS);
  CHECK_I32(positions); SAME(y, is_f32(proj));
  const int64_t B = proj.size(0);
  TORCH_CHECK(positions.numel() == B && slots.numel() == B && y.numel() == B * heads * P, "mamba_step: shapes");
  const c10::cuda::CUDAGuard guard(proj.device());
  RUN(mb::hy_mamba_step(is_f32(proj), a, positions.data_ptr<int>(), B, y.data_ptr(), cur_stream()));
}

// Prompt form: cu [B + 1], ctx [B]; conv_tiles / chunks as described in hybrid.h (chunks empty: sequential scan).
void mamba_prefill(MAMBA_ARGS, const at::Tensor& cu, const at::Tensor& ctx, const at::Tensor& conv_tiles, const OptT& chunks,
                   const OptT& first_chunk, at::Tensor& y) {
  mb::HyMamba a = make_mamba(MAMBA_PASS);
  const bool f = is_f32(proj);
  CHECK_I32(cu); CHECK_I32(ctx); CHECK_I32(conv_tiles); SAME(y, f);
  const int64_t T = proj.size(0), inner = heads * P, ch = inner + 2 * groups * N;
  TORCH_CHECK(cu.numel() == ctx.numel() + 1 && slots.numel() == ctx.numel() && y.numel() == T * inner && conv_tiles.size(1) == 4, "mamba_prefill: shapes");
  a.cu = cu.data_ptr<int>(); a.ctx = ctx.data_ptr<int>(); a.nseq = ctx.numel();
  const c10::cuda::CUDAGuard guard(proj.device());
  at::Tensor xbc = at::empty({T, ch}, proj.options());
  RUN(mb::hy_conv(f, a, conv_tiles.data_ptr<int>(), conv_tiles.size(0), xbc.data_ptr(), cur_stream()));
  if (chunks.has_value() && !f && mb::hy_chunk_scan_supported(P, N, heads, groups)) {
    CHECK_I32((*chunks)); CHECK_I32((*first_chunk));
    const int64_t n = chunks->size(0);
    TORCH_CHECK(chunks->size(1) == 4 && first_chunk->numel() == ctx.numel() + 1, "mamba_prefill: chunk tables");
    at::Tensor work = at::empty({n * heads * P * N}, state.options()), decay = at::empty({n * heads}, state.options());
    at::Tensor before = at::empty({n * heads * 2 * P * N}, proj.options());
    RUN(mb::hy_chunk_scan(a, xbc.data_ptr(), chunks->data_ptr<int>(), n, first_chunk->data_ptr<int>(), work.data_ptr<float>(),
                          decay.data_ptr<float>(), before.data_ptr(), y.data_ptr(), cur_stream()));
  } else {
    RUN(mb::hy_scan(f, a, xbc.data_ptr(), y.data_ptr(), cur_stream()));
  }
}

// ------------------------------------------------------------------------------------------------ latent attention
mb::HyLatent make_latent(int64_t heads, int64_t dim, int64_t rot, int64_t vdim, int64_t window, double scale, const at::Tensor& ukv,
                         const at::Tensor& freq, const at::Tensor& rows, const at::Tensor& table, int64_t page_size, at::Tensor& status) {
  const bool f = is_f32(ukv);
  SAME(ukv, f); SAME(rows, f); CHECK_F32(freq); CHECK_I32(table); CHECK_I32(status);
  const int64_t rank = ukv.size(1);
  TORCH_CHECK(ukv.size(0) == heads * (dim + vdim) && freq.numel() == rot / 2 && rows.size(1) >= rank + rot && rows.size(1) % 8 == 0 &&
              table.dim() == 2 && page_size > 0, "latent attention: shapes");
  mb::HyLatent a = {};
  a.heads = heads; a.dim = dim; a.rot = rot; a.vdim = vdim; a.rank = rank; a.width = rows.size(1); a.window = window; a.scale = scale;
  a.ukv = ukv.data_ptr(); a.freq = freq.data_ptr<float>(); a.rows = rows.data_ptr(); a.num_slots = rows.size(0);
  a.table = table.data_ptr<int>(); a.max_pages = table.size(1); a.page_size = page_size; a.status = status.data_ptr<int>();
  return a;
}
#define LATENT_ARGS int64_t heads, int64_t dim, int64_t rot, int64_t vdim, int64_t window, double scale, const at::Tensor &ukv, \
                    const at::Tensor &freq, const at::Tensor &rows, const at::Tensor &table, int64_t page_size, at::Tensor &status
#define LATENT_PASS heads, dim, rot, vdim, window, scale, ukv, freq, rows, table, page_size, status

void check_q(const at::Tensor& q, const at::Tensor& positions, at::Tensor& cat, const mb::HyLatent& a, bool f) {
  SAME(q, f); SAME(cat, f); CHECK_I32(positions);
  TORCH_CHECK(q.numel() == positions.numel() * a.heads * (a.dim + a.rot) && cat.dim() == 2 && cat.size(0) == positions.numel() &&
              cat.size(1) >= a.heads * a.vdim, "latent attention: queries");
}

// Any sizes, fp32 scores from the cache rows: positions [T], row_seq [T] (absent: row t is sequence t).
void latent_attend(LATENT_ARGS, const at::Tensor& q, const at::Tensor& positions, const OptT& row_seq, at::Tensor& cat) {
  const mb::HyLatent a = make_latent(LATENT_PASS);
  const bool f = is_f32(ukv);
  check_q(q, positions, cat, a, f);
  const int64_t T = positions.numel();
  if (row_seq.has_value()) { CHECK_I32((*row_seq)); TORCH_CHECK(row_seq->numel() == T, "latent_attend: row_seq"); }
  else TORCH_CHECK(table.size(0) >= T, "latent_attend: block table");
  const c10::cuda::CUDAGuard guard(q.device());
  const auto fo = q.options().dtype(at::kFloat);
  const int qld = a.rank + a.rot;
  for (int64_t t0 = 0; t0 < T; t0 += 32768) {  // (the row index is a grid dimension)
    const int64_t n = std::min<int64_t>(32768, T - t0);
    at::Tensor ql = at::empty({n, heads, qld}, fo), o = at::empty({n, heads, static_cast<int64_t>(a.rank)}, fo);
    const char* qp = static_cast<const char*>(q.data_ptr()) + t0 * heads * (dim + rot) * q.element_size();
    char* cp = static_cast<char*>(cat.data_ptr()) + t0 * cat.size(1) * cat.element_size();
    const int* pp = positions.data_ptr<int>() + t0;
    RUN(mb::hy_absorb_q(f, a, qp, pp, n, ql.data_ptr(), qld, true, cur_stream()));
    mb::HyLatent b = a;
    if (!row_seq.has_value()) b.table += t0 * a.max_pages;
    RUN(mb::hy_attend(f, mb::hy_latent_view(b), ql.data_ptr<float>(), qld, pp, row_seq.has_value() ? row_seq->data_ptr<int>() + t0 : nullptr, n,
                      o.data_ptr<float>(), nullptr, 0, cur_stream()));
    RUN(mb::hy_latent_up(f, a, o.data_ptr<float>(), nullptr, 1, n, cp, cat.size(1), cur_stream()));
  }
}

// One row per sequence on the tensor cores (bf16).
void latent_decode(LATENT_ARGS, const at::Tensor& q, const at::Tensor& positions, const at::Tensor& seq_lens, int64_t splits, at::Tensor& cat) {
  const mb::HyLatent a = make_latent(LATENT_PASS);
  check_q(q, positions, cat, a, false);
  CHECK_I32(seq_lens);
  const int64_t B = positions.numel();
  TORCH_CHECK(seq_lens.numel() == B && table.size(0) >= B, "latent_decode: shapes");
  const c10::cuda::CUDAGuard guard(q.device());
  const int64_t qld = (a.rank + a.rot + 7) / 8 * 8;
  at::Tensor ql = at::empty({B, heads, qld}, q.options());
  const auto fo = q.options().dtype(at::kFloat);
  at::Tensor o = at::empty({B, heads, splits, static_cast<int64_t>(a.rank)}, fo), ml = at::empty({B, heads, splits, 2}, fo);
  RUN(mb::hy_absorb_q(false, a, q.data_ptr(), positions.data_ptr<int>(), B, ql.data_ptr(), qld, false, cur_stream()));
  RUN(mb::hy_decode(latent_decode_view(a), ql.data_ptr(), qld, seq_lens.data_ptr<int>(), B, splits, o.data_ptr<float>(), ml.data_ptr<float>(), cur_stream()));
  RUN(mb::hy_latent_up(false, a, o.data_ptr<float>(), ml.data_ptr<float>(), splits, B, cat.data_ptr(), cat.size(1), cur_stream()));
}

// Cached rows of the ranges {sequence, first position, first output row, rows} -> [total, width].
at::Tensor gather_rows(LATENT_ARGS, const at::Tensor& ranges, int64_t total, int64_t max_rows) {
  const mb::HyLatent a = make_latent(LATENT_PASS);
  CHECK_I32(ranges);
  TORCH_CHECK(ranges.dim() == 2 && ranges.size(1) == 4, "gather_rows: ranges");
  const c10::cuda::CUDAGuard guard(rows.device());
  at::Tensor out = at::empty({total, rows.size(1)}, rows.options());
  RUN(mb::hy_gather_rows(is_f32(rows), a, ranges.data_ptr<int>(), ranges.size(0), max_rows, out.data_ptr(), cur_stream()));
  return out;
}

// Prompt attention on tcgen05 over gathered latents and the keys / values projected from them.
void latent_prefill(LATENT_ARGS, const at::Tensor& q, const at::Tensor& positions, const at::Tensor& latent, const at::Tensor& kv,
                    const at::Tensor& tiles, at::Tensor& cat) {
  const mb::HyLatent a = make_latent(LATENT_PASS);
  check_q(q, positions, cat, a, false);
  CHECK_BF16(latent); CHECK_BF16(kv); CHECK_I32(tiles);
  TORCH_CHECK(latent.size(0) == kv.size(0) && latent.size(1) == rows.size(1) && kv.size(1) == heads * (dim + vdim) && tiles.size(1) == 4, "latent_prefill: shapes");
  const c10::cuda::CUDAGuard guard(q.device());
  const int64_t T = positions.numel(), nope = dim <= 64 ? 64 : 128;
  at::Tensor qp = at::empty({T, heads * (nope + 64)}, q.options());
  RUN(mb::hy_pad_q(a, q.data_ptr(), positions.data_ptr<int>(), T, nope, 64, qp.data_ptr(), cur_stream()));
  mb::HyPrefill p = {};
  p.q = qp.data_ptr(); p.heads = heads; p.group = 1; p.dim = dim; p.vdim = vdim; p.q_pad = nope; p.window = window; p.scale = scale;
  p.kv = kv.data_ptr(); p.ctx_rows = kv.size(0); p.kv_cols = p.kv_ld = kv.size(1);
  p.k_step = dim; p.v_col = heads * dim; p.v_step = vdim;  // (every head has projected keys and values of its own)
  p.shared = latent.data_ptr(); p.rot = rot; p.shared_col = a.rank; p.shared_width = latent.size(1);
  p.status = a.status;
  const int rc = mb::hy_prefill(p, tiles.data_ptr<int>(), tiles.size(0), T, cat.data_ptr(), cat.size(1), cur_stream());
  TORCH_CHECK(rc == 0, mb::hy_prefill_last_error());
}

// ------------------------------------------------------------------------------------------------ softmax attention
// (source column, heads, dim, rotated dims, frequencies, unit norm, scale, destination, first column, columns per head, zero columns
// after the last head, destination rows by slot)
typedef std::tuple<int64_t, int64_t, int64_t, int64_t, OptT, bool, double, at::Tensor, int64_t, int64_t, int64_t, bool> HeadOp;

// For many rows: room for the angles of every operation, one table for operations that turn alike.
at::Tensor add_turns(mb::HyHeadRows& a, int64_t T, const at::Tensor& like) {
  at::Tensor work;
  if (T <= 512) return work;
  int64_t total = 0, at[3];
  int same[3];
  for (int i = 0; i < a.n; ++i) {
    same[i] = i;
    for (int j = 0; j < i; ++j)
      if (a.op[j].freq == a.op[i].freq && a.op[j].rot == a.op[i].rot) { same[i] = j; break; }
    at[i] = same[i] < i ? at[same[i]] : total;
    if (same[i] == i) total += T * (a.op[i].rot / 2);
  }
  work = at::empty({total, 2}, like.options().dtype(at::kFloat));
  for (int i = 0; i < a.n; ++i) {
    a.turns[i] = reinterpret_cast<float2*>(work.data_ptr<float>()) + at[i];
    a.fill[i] = same[i] == i && a.op[i].rot > 0;
  }
  return work;
}

void head_rows(const at::Tensor& proj, const at::Tensor& positions, const OptT& slots, double eps, at::Tensor& status, const std::vector<HeadOp>& ops) {
  const bool f = is_f32(proj);
  SAME(proj, f); CHECK_I32(positions); CHECK_I32(status);
  TORCH_CHECK(proj.dim() == 2 && positions.numel() == proj.size(0) && ops.size() >= 1 && ops.size() <= 3, "head_rows: shapes");
  const int64_t T = proj.size(0);
  mb::HyHeadRows a = {};
  a.n = ops.size(); a.proj = proj.data_ptr(); a.ld = proj.size(1); a.positions = positions.data_ptr<int>(); a.eps = eps; a.status = status.data_ptr<int>();
  if (slots.has_value()) { CHECK_I32((*slots)); TORCH_CHECK(slots->numel() == T, "head_rows: slots"); a.slots = slots->data_ptr<int>(); }
  for (size_t i = 0; i < ops.size(); ++i) {
    mb::HyHeadOp& o = a.op[i];
    at::Tensor dst;
    OptT freq;
    std::tie(o.src, o.heads, o.dim, o.rot, freq, o.unit, o.scale, dst, o.col, o.pitch, o.tail, o.by_slot) = ops[i];
    TORCH_CHECK(dst.is_cuda() && dst.is_contiguous() && dst.dim() == 2 && (dst.scalar_type() == at::kFloat || dst.scalar_type() == proj.scalar_type()),
                "head_rows: destination");
    TORCH_CHECK(o.src >= 0 && o.heads >= 1 && o.src + o.heads * o.dim <= proj.size(1) && o.rot % 2 == 0 && o.rot >= 0 && o.rot <= o.dim && o.pitch >= o.dim &&
                o.tail >= 0 && o.col >= 0 && o.col + o.heads * o.pitch + o.tail <= dst.size(1), "head_rows: columns");
    if (o.rot > 0) { TORCH_CHECK(freq.has_value() && freq->numel() >= o.rot / 2, "head_rows: frequencies"); CHECK_F32((*freq)); o.freq = freq->data_ptr<float>(); }
    o.dst = dst.data_ptr(); o.ld = dst.size(1);
    o.f32 = !f && dst.scalar_type() == at::kFloat;
    if (o.by_slot) {
      TORCH_CHECK(slots.has_value() && (a.num_slots == 0 || a.num_slots == dst.size(0)), "head_rows: cache rows");
      a.num_slots = dst.size(0);
    } else {
      TORCH_CHECK(dst.size(0) == T, "head_rows: rows");
    }
  }
  const c10::cuda::CUDAGuard guard(proj.device());
  const at::Tensor work = add_turns(a, T, proj);
  RUN(mb::hy_head_rows(f, a, T, cur_stream()));
}

mb::HyAttend make_attend(int64_t heads, int64_t kv_heads, int64_t dim, int64_t vdim, double scale, const OptT& sink, const at::Tensor& rows,
                         const at::Tensor& table, int64_t page_size, at::Tensor& status) {
  const bool f = is_f32(rows);
  SAME(rows, f); CHECK_I32(table); CHECK_I32(status);
  TORCH_CHECK(kv_heads >= 1 && heads >= 1 && heads % kv_heads == 0 && rows.dim() == 2 && rows.size(1) >= kv_heads * (dim + vdim) && table.dim() == 2 && page_size > 0,
              "attention: shapes");
  mb::HyAttend a = {};
  a.rows = rows.data_ptr(); a.num_slots = rows.size(0); a.width = rows.size(1);
  a.table = table.data_ptr<int>(); a.max_pages = table.size(1); a.page_size = page_size; a.status = status.data_ptr<int>();
  a.heads = heads; a.group = heads / kv_heads; a.kd = dim; a.vd = vdim;
  a.k_step = dim; a.v_col = kv_heads * dim; a.v_step = vdim;
  a.scale = scale;
  if (sink.has_value()) { SAME((*sink), f); TORCH_CHECK(sink->numel() == heads, "attention: sinks"); a.sink = sink->data_ptr(); }
  return a;
}
#define ATTN_ARGS int64_t heads, int64_t kv_heads, int64_t dim, int64_t vdim, double scale, const OptT &sink, const at::Tensor &rows, \
                  const at::Tensor &table, int64_t page_size, at::Tensor &status
#define ATTN_PASS heads, kv_heads, dim, vdim, scale, sink, rows, table, page_size, status

bool attn_decode_supported(int64_t heads, int64_t kv_heads, int64_t dim, int64_t vdim, int64_t width) {
  mb::HyAttend a = {};
  a.heads = heads; a.group = heads / kv_heads; a.kd = a.k_step = dim; a.vd = a.v_step = vdim; a.v_col = kv_heads * dim; a.width = width;
  return mb::hy_decode_supported(a);
}

// Any sizes, fp32 scores from the cache rows: q [T, heads, dim] fp32, positions [T], row_seq [T] (absent: row t is sequence t).
void attn_plain(ATTN_ARGS, const at::Tensor& q, const at::Tensor& positions, const OptT& row_seq, at::Tensor& out) {
  const mb::HyAttend a = make_attend(ATTN_PASS);
  const bool f = is_f32(rows);
  CHECK_F32(q); CHECK_I32(positions); SAME(out, f);
  const int64_t T = positions.numel();
  TORCH_CHECK(q.numel() == T * heads * dim && out.dim() == 2 && out.size(0) == T && out.size(1) >= heads * vdim, "attn_plain: shapes");
  if (row_seq.has_value()) { CHECK_I32((*row_seq)); TORCH_CHECK(row_seq->numel() == T, "attn_plain: row_seq"); }
  else TORCH_CHECK(table.size(0) >= T, "attn_plain: block table");
  const c10::cuda::CUDAGuard guard(q.device());
  for (int64_t t0 = 0; t0 < T; t0 += 32768) {  // (the row index is a grid dimension)
    const int64_t n = std::min<int64_t>(32768, T - t0);
    mb::HyAttend b = a;
    if (!row_seq.has_value()) b.table += t0 * a.max_pages;
    RUN(mb::hy_attend(f, b, q.data_ptr<float>() + t0 * heads * dim, dim, positions.data_ptr<int>() + t0, row_seq.has_value() ? row_seq->data_ptr<int>() + t0 : nullptr,
                      n, nullptr, static_cast<char*>(out.data_ptr()) + t0 * out.size(1) * out.element_size(), out.size(1), cur_stream()));
  }
}

// One row per sequence on the tensor cores (bf16): q [B, heads, dim].
void attn_decode(ATTN_ARGS, const at::Tensor& q, const at::Tensor& seq_lens, int64_t splits, at::Tensor& out) {
  const mb::HyAttend a = make_attend(ATTN_PASS);
  SAME(rows, false); SAME(q, false); SAME(out, false); CHECK_I32(seq_lens);
  const int64_t B = seq_lens.numel();
  TORCH_CHECK(q.numel() == B * heads * dim && table.size(0) >= B && out.dim() == 2 && out.size(0) == B && out.size(1) >= heads * vdim, "attn_decode: shapes");
  const c10::cuda::CUDAGuard guard(q.device());
  const auto fo = q.options().dtype(at::kFloat);
  at::Tensor o = at::empty({B, heads, splits, vdim}, fo), ml = at::empty({B, heads, splits, 2}, fo);
  RUN(mb::hy_decode(a, q.data_ptr(), dim, seq_lens.data_ptr<int>(), B, splits, o.data_ptr<float>(), ml.data_ptr<float>(), cur_stream()));
  RUN(mb::hy_decode_merge(false, a, o.data_ptr<float>(), ml.data_ptr<float>(), splits, B, out.data_ptr(), out.size(1), cur_stream()));
}

// Prompt attention on tcgen05: q [T, heads, q_pad], the rows of the ranges {sequence, first position, first output row, rows} gathered.
void attn_prefill(ATTN_ARGS, const at::Tensor& q, int64_t q_pad, const at::Tensor& ranges, int64_t total, int64_t max_rows, const at::Tensor& tiles,
                  at::Tensor& out) {
  const mb::HyAttend a = make_attend(ATTN_PASS);
  SAME(rows, false); SAME(q, false); SAME(out, false); CHECK_I32(ranges); CHECK_I32(tiles);
  const int64_t T = out.size(0);
  TORCH_CHECK(q.numel() == T * heads * q_pad && out.size(1) >= heads * vdim && ranges.size(1) == 4 && tiles.size(1) == 4, "attn_prefill: shapes");
  const c10::cuda::CUDAGuard guard(q.device());
  at::Tensor kv = at::empty({total, rows.size(1)}, rows.options());
  RUN(mb::hy_gather_rows(false, a, ranges.data_ptr<int>(), ranges.size(0), max_rows, kv.data_ptr(), cur_stream()));
  mb::HyPrefill p = {};
  p.q = q.data_ptr(); p.heads = heads; p.group = a.group; p.dim = dim; p.vdim = vdim; p.q_pad = q_pad; p.scale = scale;
  p.kv = kv.data_ptr(); p.ctx_rows = total; p.kv_cols = p.kv_ld = rows.size(1);
  p.k_step = a.k_step; p.v_col = a.v_col; p.v_step = a.v_step;
  p.sink = a.sink; p.status = a.status;
  const int rc = mb::hy_prefill(p, tiles.data_ptr<int>(), tiles.size(0), T, out.data_ptr(), out.size(1), cur_stream());
  TORCH_CHECK(rc == 0, mb::hy_prefill_last_error());
}
bool attn_prefill_supported(int64_t kv_heads, int64_t dim, int64_t vdim, int64_t width) {
  return (kv_heads * dim) % 8 == 0 && width % 8 == 0 && mb::hy_prefill_supported(dim, 0, vdim, 0, 0);
}

// ------------------------------------------------------------------------------------------------ linear attention
// columns: first column of values, keys, queries, output gates, decay input (-1 without one)
#define LIN_ARGS at::Tensor &proj, const std::vector<int64_t> &columns, int64_t heads, int64_t P, int64_t N, double q_scale, double k_scale, int64_t rot, \
                 const OptT &freq, const OptT &decay_m1, const OptT &log2_decay, const OptT &a2, const OptT &a2_bias, double inv_tau, const OptT &norm,  \
                 double eps, at::Tensor &state, const at::Tensor &slots, at::Tensor &status
#define LIN_PASS proj, columns, heads, P, N, q_scale, k_scale, rot, freq, decay_m1, log2_decay, a2, a2_bias, inv_tau, norm, eps, state, slots, status

mb::HyLinear make_linear(LIN_ARGS) {
  const bool f = is_f32(proj);
  SAME(proj, f); CHECK_F32(state); CHECK_I32(slots); CHECK_I32(status);
  TORCH_CHECK(proj.dim() == 2 && columns.size() == 5 && heads >= 1 && P >= 1 && N >= 1, "linear attention: shapes");
  mb::HyLinear a = {};
  a.proj = proj.data_ptr(); a.ld = proj.size(1);
  a.v = columns[0]; a.k = columns[1]; a.q = columns[2]; a.g = columns[3]; a.u = columns[4];
  a.heads = heads; a.P = P; a.N = N; a.q_scale = q_scale; a.k_scale = k_scale; a.rot = rot; a.inv_tau = inv_tau; a.eps = eps;
  const int64_t wide[4] = {a.v + heads * P, a.k + heads * N, a.q + heads * N, a.g + heads * P};
  for (int64_t w : wide) TORCH_CHECK(w <= a.ld, "linear attention: columns");
  if (rot > 0) {
    TORCH_CHECK(freq.has_value() && freq->numel() == rot / 2 && rot % 2 == 0 && rot <= N, "linear attention: frequencies");
    CHECK_F32((*freq));
    a.freq = freq->data_ptr<float>();
  }
  if (a2.has_value()) {
    SAME((*a2), f); TORCH_CHECK(a2_bias.has_value(), "linear attention: decay bias"); SAME((*a2_bias), f);
    a.rank = a2->size(1);
    TORCH_CHECK(a.rank >= 1 && a2->size(0) == heads * N && a2_bias->numel() == heads * N && a.u >= 0 && a.u + a.rank <= a.ld, "linear attention: decay");
    a.a2 = a2->data_ptr(); a.a2_bias = a2_bias->data_ptr();
  } else {
    TORCH_CHECK(decay_m1.has_value() && log2_decay.has_value(), "linear attention: decay");
    CHECK_F32((*decay_m1)); CHECK_F32((*log2_decay));
    TORCH_CHECK(decay_m1->numel() == heads && log2_decay->numel() == heads, "linear attention: decay");
    a.decay_m1 = decay_m1->data_ptr<float>(); a.log2_decay = log2_decay->data_ptr<float>();
  }
  if (norm.has_value()) { SAME((*norm), f); TORCH_CHECK(norm->numel() == P, "linear attention: norm"); a.norm = norm->data_ptr(); }
  TORCH_CHECK(state.dim() == 4 && state.size(1) == heads && state.size(2) == P && state.size(3) == N, "linear attention: state");
  a.state = state.data_ptr<float>(); a.sequences = state.size(0);
  a.slots = slots.data_ptr<int>(); a.status = status.data_ptr<int>();
  return a;
}
void check_lin_out(const at::Tensor& proj, const at::Tensor& out, const mb::HyLinear& a) {
  SAME(out, is_f32(proj));
  TORCH_CHECK(out.dim() == 2 && out.size(0) == proj.size(0) && out.size(1) >= a.heads * a.P, "linear attention: output");
}

void linear_step(LIN_ARGS, const at::Tensor& positions, at::Tensor& out) {
  const mb::HyLinear a = make_linear(LIN_PASS);
  check_lin_out(proj, out, a);
  CHECK_I32(positions);
  const int64_t B = proj.size(0);
  TORCH_CHECK(positions.numel() == B && slots.numel() == B, "linear_step: shapes");
  const c10::cuda::CUDAGuard guard(proj.device());
  RUN(mb::hy_linear_step(is_f32(proj), a, positions.data_ptr<int>(), B, out.data_ptr(), out.size(1), cur_stream()));
}

// Prompt form: cu [B + 1], ctx [B]; rotates queries and keys in place. chunks as in mamba_prefill (absent: sequential scan).
void linear_prefill(LIN_ARGS, const at::Tensor& positions, const at::Tensor& cu, const at::Tensor& ctx, const OptT& chunks, const OptT& first_chunk, at::Tensor& out) {
  mb::HyLinear a = make_linear(LIN_PASS);
  check_lin_out(proj, out, a);
  const bool f = is_f32(proj);
  CHECK_I32(positions); CHECK_I32(cu); CHECK_I32(ctx);
  const int64_t T = proj.size(0);
  TORCH_CHECK(positions.numel() == T && cu.numel() == ctx.numel() + 1 && slots.numel() == ctx.numel(), "linear_prefill: shapes");
  a.cu = cu.data_ptr<int>(); a.ctx = ctx.data_ptr<int>(); a.nseq = ctx.numel();
  const c10::cuda::CUDAGuard guard(proj.device());
  const cudaStream_t s = cur_stream();
  if (rot > 0 || k_scale != 1.0) {
    mb::HyHeadRows r = {};
    r.proj = proj.data_ptr(); r.ld = a.ld; r.positions = positions.data_ptr<int>(); r.status = a.status;
    const int cols[2] = {a.q, a.k};
    for (int i = 0; i < 2; ++i) {
      mb::HyHeadOp& o = r.op[r.n++];
      o.src = o.col = cols[i]; o.heads = a.heads; o.dim = o.pitch = a.N; o.rot = a.rot; o.freq = a.freq;
      o.scale = i == 0 ? 1.f : a.k_scale;
      o.dst = proj.data_ptr(); o.ld = a.ld;
    }
    const at::Tensor work = add_turns(r, T, proj);
    RUN(mb::hy_head_rows(f, r, T, s));
  }
  at::Tensor y = at::empty({T, heads * P}, proj.options()), gate;
  const bool by_channel = a.rank > 0;
  const bool fast = chunks.has_value() && !f && (by_channel ? mb::hy_linear_chunks_supported(P, N) : q_scale == 1.0 && mb::hy_chunk_scan_supported(P, N, heads, heads));
  if (by_channel) {
    gate = at::empty({T, heads * N}, state.options());
    RUN(mb::hy_linear_gate(f, a, fast ? chunks->data_ptr<int>() : nullptr, fast ? chunks->size(0) : 0, T, gate.data_ptr<float>(), s));
  }
  if (fast) {
    CHECK_I32((*chunks)); CHECK_I32((*first_chunk));
    const int64_t n = chunks->size(0);
    TORCH_CHECK(chunks->size(1) == 4 && first_chunk->numel() == ctx.numel() + 1, "linear_prefill: chunk tables");
    at::Tensor work = at::empty({n * heads * P * N}, state.options()), before = at::empty({n * heads * 2 * P * N}, proj.options());
    at::Tensor decay = at::empty({n * heads * (by_channel ? 2 * N : 1)}, state.options());
    if (by_channel) {
      at::Tensor far = at::empty({n * heads}, slots.options());
      RUN(mb::hy_linear_chunks(a, gate.data_ptr<float>(), chunks->data_ptr<int>(), n, first_chunk->data_ptr<int>(), work.data_ptr<float>(), decay.data_ptr<float>(),
                               far.data_ptr<int>(), before.data_ptr(), y.data_ptr(), s));
    } else {
      mb::HyMamba m = {};
      m.proj = a.proj; m.ld = m.xld = a.ld; m.x_col = a.v; m.b_col = a.k; m.c_col = a.q;
      m.log2_decay = a.log2_decay;
      m.heads = m.groups = a.heads; m.P = a.P; m.N = a.N;
      m.state = a.state; m.sequences = a.sequences; m.cu = a.cu; m.ctx = a.ctx; m.slots = a.slots; m.nseq = a.nseq; m.status = a.status;
      RUN(mb::hy_chunk_scan(m, proj.data_ptr(), chunks->data_ptr<int>(), n, first_chunk->data_ptr<int>(), work.data_ptr<float>(), decay.data_ptr<float>(),
                            before.data_ptr(), y.data_ptr(), s));
    }
  } else {
    RUN(mb::hy_linear_scan(f, a, by_channel ? gate.data_ptr<float>() : nullptr, y.data_ptr(), s));
  }
  RUN(mb::hy_linear_tail(f, a, y.data_ptr(), T, out.data_ptr(), out.size(1), s));
}

// ------------------------------------------------------------------------------------------------ sequential blocks
void gated_act(const at::Tensor& proj, int64_t gate, int64_t up, int64_t ff, bool relu, at::Tensor& out) {
  const bool f = is_f32(proj);
  SAME(proj, f); SAME(out, f);
  TORCH_CHECK(proj.dim() == 2 && out.dim() == 2 && proj.size(0) == out.size(0) && gate + ff <= proj.size(1) && up + ff <= proj.size(1) && ff <= out.size(1), "gated_act: shapes");
  const c10::cuda::CUDAGuard guard(proj.device());
  RUN(mb::hy_gated_act(f, proj.data_ptr(), proj.size(1), gate, up, ff, relu ? 1 : 0, proj.size(0), out.data_ptr(), out.size(1), cur_stream()));
}

void embed_layer_norm(const at::Tensor& tokens, const at::Tensor& table, const at::Tensor& next, at::Tensor& x, at::Tensor& h, double eps, at::Tensor& status) {
  const bool f = is_f32(table);
  CHECK_I32(tokens); CHECK_F32(x); CHECK_I32(status);
  SAME(table, f); SAME(next, f); SAME(h, f);
  const int64_t T = tokens.numel(), H = table.size(1);
  TORCH_CHECK(next.numel() == H && x.numel() == T * H && h.numel() == T * H, "embed_layer_norm: shapes");
  mb::HySandwich a = {};
  a.x = x.data_ptr<float>(); a.tokens = tokens.data_ptr<int>(); a.table = table.data_ptr(); a.V = table.size(0);
  a.next = next.data_ptr(); a.h = h.data_ptr(); a.H = H; a.eps = eps; a.status = status.data_ptr<int>();
  const c10::cuda::CUDAGuard guard(table.device());
  RUN(mb::hy_sandwich(f, a, T, cur_stream()));
}

// x += layernorm(y) * post, h = layernorm(x) * next; with y2: y = (rms(y) w1 + rms(y2) w2) / 2 first.
void sandwich(at::Tensor& x, const at::Tensor& y, const OptT& y2, const OptT& w1, const OptT& w2, const at::Tensor& post, const at::Tensor& next, at::Tensor& h, double eps) {
  const bool f = is_f32(post);
  CHECK_F32(x); CHECK_F32(y);
  SAME(post, f); SAME(next, f); SAME(h, f);
  const int64_t T = x.size(0), H = x.size(1);
  TORCH_CHECK(y.numel() == T * H && post.numel() == H && next.numel() == H && h.numel() == T * H, "sandwich: shapes");
  mb::HySandwich a = {};
  a.x = x.data_ptr<float>(); a.y = y.data_ptr<float>(); a.post = post.data_ptr(); a.next = next.data_ptr(); a.h = h.data_ptr(); a.H = H; a.eps = eps;
  if (y2.has_value()) {
    CHECK_F32((*y2)); TORCH_CHECK(w1.has_value() && w2.has_value() && y2->numel() == T * H, "sandwich: second output");
    SAME((*w1), f); SAME((*w2), f);
    TORCH_CHECK(w1->numel() == H && w2->numel() == H, "sandwich: weights");
    a.y2 = y2->data_ptr<float>(); a.w1 = w1->data_ptr(); a.w2 = w2->data_ptr();
  }
  const c10::cuda::CUDAGuard guard(x.device());
  RUN(mb::hy_sandwich(f, a, T, cur_stream()));
}

}  // namespace

PYBIND11_MODULE(_hybrid, m) {
  register_serving(m);
  m.def("embed_norm", &embed_norm);
  m.def("mamba_tail", &mamba_tail);
  m.def("latent_in", &latent_in);
  m.def("side_fused", &side_fused);
  m.def("side_gate", &side_gate);
  m.def("side_finish", &side_finish);
  m.def("cast_rows", &cast_rows);
  m.def("mamba_step", &mamba_step);
  m.def("mamba_prefill", &mamba_prefill);
  m.def("latent_attend", &latent_attend);
  m.def("latent_decode", &latent_decode);
  m.def("gather_rows", &gather_rows);
  m.def("latent_prefill", &latent_prefill);
  m.def("head_rows", &head_rows);
  m.def("attn_plain", &attn_plain);
  m.def("attn_decode", &attn_decode);
  m.def("attn_decode_supported", &attn_decode_supported);
  m.def("attn_prefill", &attn_prefill);
  m.def("attn_prefill_supported", &attn_prefill_supported);
  m.def("linear_step", &linear_step);
  m.def("linear_prefill", &linear_prefill);
  m.def("linear_chunks_supported", &mb::hy_linear_chunks_supported);
  m.def("gated_act", &gated_act);
  m.def("embed_layer_norm", &embed_layer_norm);
  m.def("sandwich", &sandwich);
  m.def("chunk_scan_supported", &mb::hy_chunk_scan_supported);
  m.def("latent_decode_supported", &latent_decode_supported);
  m.def("latent_prefill_supported", &mb::hy_prefill_supported);
  m.attr("CHUNK") = mb::HY_CHUNK;
}
