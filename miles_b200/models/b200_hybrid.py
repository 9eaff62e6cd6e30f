"""sm_100a execution of models with a layer plan (``models/layer_plan.py``), for prompts and for decoding.

A parallel layer is two large products with fused kernels between them:

    proj = [mixer input | gate | up] h             one product over everything that reads the normed input
    mixer kernels on proj                          (recurrence or latent attention, see csrc/mamba2.cu, latent_attention.cu)
    cat  = [mixer output | silu(gate) * up]        written by the mixers' last kernels
    x   += [o | down] cat                          one product over everything that writes the residual, fp32
    x   += rmsnorm(proj(gelu(gate x) * e)) * norm  per-layer token input, ending in the next layer's norm

A sequential layer has one product in front of and one behind each mixer or feed-forward, and one kernel per sublayer that norms
its output, adds it to the residual and norms that for whatever reads it next:

    proj = [everything the mixer reads] h
    out  = mixer kernels on proj                   (csrc/linear_attention.cu, cached_attention.cu, cached_prefill.cu)
    y    = o out (fp32; two of them where two mixers run side by side)
    x   += norm(y), h = norm(x)                    (csrc/sequential_ops.cu)

bf16 stores run the products on the tcgen05 GEMM (few rows: the weight-streaming kernel), prompts through the chunked
recurrence and the tcgen05 attention. fp32 stores run the same layer code with 32-bit products and the plain kernels of any
size. Head sizes the tensor-core kernels do not take fall to those plain kernels too, in bf16.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn.functional as F

from ..ops import _ext
from ..ops.attention import TILE_Q
from ..ops.reference import pair_frequencies
from .config import ModelConfig
from .layer_plan import LinearAttention, Mamba2, Parallel
from .params import ParamStore
from .torch_hybrid import TorchHybrid
from .torch_impl import InferMeta

CONV_TILE = 32
SMALL_T = 32       # rows up to which products stream the weights instead of filling tcgen05 tiles
FUSED_SIDE_T = 16  # rows up to which the per-layer token input is one kernel


class B200Hybrid(TorchHybrid):
    def __init__(self, cfg: ModelConfig, store: ParamStore):
        super().__init__(cfg, store)
        assert store.device.type == "cuda" and store.dtype in (torch.bfloat16, torch.float32)
        self.C = _ext.load_hybrid()
        self.f32 = store.dtype == torch.float32
        self.status = torch.zeros(1, dtype=torch.int32, device=self.dev)
        self.launches = 0
        self.freq = {}
        self.fixed_decay = {}  # (layer, side) -> decays - 1 and their base-2 logarithms
        for i, l in enumerate(cfg.plan.layers):
            for side, m in l.mixer.sides() if isinstance(l.mixer, Parallel) else [("", l.mixer)]:
                r = getattr(m, "rotary", None)
                if r is not None:
                    self.freq[(r.base, r.dims)] = pair_frequencies(r.dims, r.base, self.dev)
                if isinstance(m, LinearAttention) and m.decay is not None:
                    d = torch.tensor(m.decay, dtype=torch.float64)
                    self.fixed_decay[(i, side)] = ((d - 1).float().to(self.dev), d.log2().clamp(min=-1e4).float().to(self.dev))
        self.sms = torch.cuda.get_device_properties(self.dev).multi_processor_count
        self.plain = False  # True: the kernels of any size everywhere (what the fast ones are checked against)

    # ------------------------------------------------------------------ products
    def linear(self, x, w, out_dtype: Optional[torch.dtype] = None):
        """x [T, K] . w [N, K]^T."""
        out_dtype = out_dtype or self.store.dtype
        if self.f32:
            return F.linear(x, w)
        T, (N, K) = x.shape[0], w.shape
        if K % 8:  # rows the tensor maps cannot describe: the vendor product
            return torch.mm(x, w.t(), out_dtype=out_dtype) if out_dtype != x.dtype else F.linear(x, w)
        out = torch.empty(T, N, dtype=out_dtype, device=x.device)
        self.launches += 1
        if T <= SMALL_T and N % 16 == 0 and K % 32 == 0 and (T <= 8 or N * K * 2 < (48 << 20)) and x.is_contiguous():
            self.C.small_gemv(x, None, 0.0, w, None, out, self.status)
        else:
            self.C.gemm(x, w, out, False, False, False, 0, self.status)
        return out

    def check_status(self) -> None:
        code = int(self.status.item())
        if code != 0:
            self.status.zero_()
            raise RuntimeError(f"a miles_b200 kernel reported error status {code} (1-5: a bounded wait expired, 8 / 9: length or page "
                               "outside the cache, 10: token id outside the vocabulary, 11: state row outside the cache)")

    # ------------------------------------------------------------------ launch tables of a prompt pass
    def _upload(self, rows) -> torch.Tensor:
        t = torch.tensor(rows, dtype=torch.int32).view(-1, 4)
        return t.pin_memory().to(self.dev, non_blocking=True)

    def _tables(self, meta: InferMeta) -> dict:
        """Convolution tiles and chunks of a pass: {sequence, first row, rows, index in the sequence}."""
        t = meta.tables
        if "chunks" not in t:
            cu, q = meta.cu_list, self.C.CHUNK
            conv, chunks, first = [], [], [0]
            for b in range(len(cu) - 1):
                n = cu[b + 1] - cu[b]
                conv += [(b, cu[b] + r, min(CONV_TILE, n - r), 0) for r in range(0, n, CONV_TILE)]
                chunks += [(b, cu[b] + r, min(q, n - r), r // q) for r in range(0, n, q)]
                first.append(len(chunks))
            t["conv"], t["chunks"] = self._upload(conv), self._upload(chunks)
            t["first"] = torch.tensor(first, dtype=torch.int32).pin_memory().to(self.dev, non_blocking=True)
        return t

    def _attn_tables(self, meta: InferMeta, window: int):
        """(gather ranges, total rows, longest range, attention tiles) of a pass: each sequence's visible keys, from the
        first one its first new token sees, are gathered into consecutive rows."""
        key = ("attn", window)
        if key not in meta.tables:
            cu, ranges, tiles, at, longest = meta.cu_list, [], [], 0, 0
            for b, ctx in enumerate(meta.ctx_list):
                n = cu[b + 1] - cu[b]
                lo = max(0, ctx - window + 1) if window else 0
                ranges.append((b, lo, at, ctx + n - lo))
                tiles += [(cu[b] + r, min(TILE_Q, n - r), at, ctx - lo + r) for r in range(0, n, TILE_Q)]
                at += ctx + n - lo
                longest = max(longest, ctx + n - lo)
            tiles.sort(key=lambda r: -min(r[3] + r[1], (window or 1 << 30) + TILE_Q))  # long tiles first
            meta.tables[key] = (self._upload(ranges), at, longest, self._upload(tiles))
        return meta.tables[key]

    def _row_seq(self, meta: InferMeta):
        if "row_seq" not in meta.tables:
            n = meta.cu_seqlens[1:] - meta.cu_seqlens[:-1]
            meta.tables["row_seq"] = torch.repeat_interleave(torch.arange(n.numel(), dtype=torch.int32, device=self.dev), n.long(),
                                                             output_size=meta.cu_list[-1])
        return meta.tables["row_seq"]

    # ------------------------------------------------------------------ mixers
    def _mamba2(self, i, proj, cat, ff, meta, cache, positions):
        m, P, p, C = self.plan.layers[i].mixer, self.store.params, f"layers.{i}.mix.", self.C
        ring, state = cache
        args = (proj, m.heads, m.vdim, m.state, m.groups, P[p + "conv.weight"], P[p + "conv.bias"], P[p + "dt_bias"], P[p + "A_log"],
                P[p + "D"], ring, state, meta.state_slots, self.status)
        y = torch.empty(proj.shape[0], m.inner, dtype=proj.dtype, device=self.dev)
        if meta.is_prefill:
            t = self._tables(meta)
            fast = not self.plain
            C.mamba_prefill(*args, meta.cu_seqlens, meta.ctx_lens, t["conv"], t["chunks"] if fast else None, t["first"] if fast else None, y)
            self.launches += 5
        else:
            C.mamba_step(*args, positions, y)
            self.launches += 1
        C.mamba_tail(y, P[p + "norm.weight"], m.norm_groups, self.plan.eps, proj, cat, *ff)
        self.launches += 1

    def _latent_attention(self, i, proj, cat, ff, meta, cache, positions):
        m, P, p, C = self.plan.layers[i].mixer, self.store.params, f"layers.{i}.mix.", self.C
        segs, rows = self.in_segs[i], cache[0]
        freq = self.freq[(m.rotary.base, m.rotary.dims)]
        cq = torch.empty(proj.shape[0], m.q_rank, dtype=proj.dtype, device=self.dev)
        own = m.kv_from is None
        C.latent_in(proj, cat, *ff[:3], m.out_dim, ff[3], segs["mix.dq"].start, P[p + "q_norm.weight"],
                    segs["mix.dkv"].start if own else -1, m.rot_dim, P[p + "kv_norm.weight"] if own else None, freq, positions,
                    meta.slot_mapping if own else None, cq, rows if own else None, self.plan.eps, self.status)
        q = self.linear(cq, P[p + "uq.weight"])
        ukv = P[p + "ukv.weight"]
        args = (m.heads, m.dim, m.rot_dim, m.vdim, m.window, m.scale, ukv, freq, rows, meta.block_table, meta.page_size, self.status)
        fast = not self.f32 and not self.plain
        width = rows.shape[1]
        self.launches += 4
        if not meta.is_prefill:
            if fast and C.latent_decode_supported(m.heads, m.kv_rank, m.rot_dim, width):
                B = q.shape[0]
                groups = (m.heads + 15) // 16 if m.heads <= 16 else (m.heads + 31) // 32
                longest = meta.block_table.shape[1] * meta.page_size
                if m.window:
                    longest = min(longest, m.window)
                splits = self._decode_splits(B, groups, longest)
                C.latent_decode(*args, q, positions, meta.seq_lens, splits, cat)
            else:
                C.latent_attend(*args, q, positions, None, cat)
        elif fast and C.latent_prefill_supported(m.dim, m.rot_dim, m.vdim, m.kv_rank, width):
            ranges, total, longest, tiles = self._attn_tables(meta, m.window)
            latent = C.gather_rows(*args, ranges, total, longest)
            kv = self.linear(latent[:, :m.kv_rank], ukv)
            C.latent_prefill(*args, q, positions, latent, kv, tiles, cat)
        else:
            C.latent_attend(*args, q, positions, self._row_seq(meta), cat)

    def _rows_for(self, T: int, width: int, used: int):
        """Input rows of a product with ``width`` columns, of which the mixer fills ``used``."""
        return (torch.empty if used == width else torch.zeros)(T, width, dtype=self.store.dtype, device=self.dev)

    def _decode_splits(self, B: int, groups: int, longest: int, per_sm: int = 1) -> int:
        """Parts the keys of a decode step are cut into, so that ``per_sm`` blocks find work on every SM."""
        return max(1, min(per_sm * self.sms // max(1, B * groups), (longest + 63) // 64, 32))

    def _attention(self, i, m, side, proj, positions, meta, rows):
        """Softmax attention over cached key / value heads; keys and values of ``proj`` go to their cache rows."""
        P, C, T = self.store.params, self.C, proj.shape[0]
        col = {n: self.in_segs[i][f"mix.{side}{n}"].start for n in ("q", "k", "v")}
        r = m.rotary
        rot, freq = (r.dims, self.freq[(r.base, r.dims)]) if r is not None else (0, None)
        fast = not self.f32 and not self.plain
        if meta.is_prefill:
            fast = fast and C.attn_prefill_supported(m.kv_heads, m.dim, m.vdim, rows.shape[1])
        else:
            fast = fast and C.attn_decode_supported(m.heads, m.kv_heads, m.dim, m.vdim, rows.shape[1])
        pitch = (64 if m.dim <= 64 else 128) if fast and meta.is_prefill else m.dim
        q = torch.empty(T, m.heads * pitch, dtype=self.store.dtype if fast else torch.float32, device=self.dev)
        nk, nv = m.kv_heads * m.dim, m.kv_heads * m.vdim
        C.head_rows(proj, positions, meta.slot_mapping, self.plan.eps, self.status,
                    [(col["q"], m.heads, m.dim, rot, freq, m.unit_qk, 1.0, q, 0, pitch, 0, False),
                     (col["k"], m.kv_heads, m.dim, rot, freq, m.unit_qk, 1.0, rows, 0, m.dim, 0, True),
                     (col["v"], m.kv_heads, m.vdim, 0, None, False, 1.0, rows, nk, m.vdim, rows.shape[1] - nk - nv, True)])
        out = self._rows_for(T, P[f"layers.{i}.{side}o.weight"].shape[1], m.out_dim)
        args = (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, P[f"layers.{i}.mix.{side}sink"] if m.sink else None, rows, meta.block_table,
                meta.page_size, self.status)
        self.launches += 3
        if not fast:
            C.attn_plain(*args, q, positions, self._row_seq(meta) if meta.is_prefill else None, out)
        elif meta.is_prefill:
            ranges, total, longest, tiles = self._attn_tables(meta, 0)
            C.attn_prefill(*args, q, pitch, ranges, total, longest, tiles, out)
        else:
            per_head = m.heads // m.kv_heads
            groups = m.kv_heads * ((per_head + 15) // 16 if per_head <= 16 else (per_head + 31) // 32)
            C.attn_decode(*args, q, meta.seq_lens, self._decode_splits(T, groups, meta.block_table.shape[1] * meta.page_size, 3), out)
        return out

    def _linear_attention(self, i, m, side, proj, positions, meta, state):
        P, C, p = self.store.params, self.C, f"layers.{i}.mix.{side}"
        segs = self.in_segs[i]
        cols = [segs[f"mix.{side}{n}"].start for n in ("v", "k", "q", "g")] + [segs[f"mix.{side}a1"].start if m.rank else -1]
        fixed = self.fixed_decay.get((i, side), (None, None))
        s = m.dim ** -0.5
        rot, freq = (m.rotary.dims, self.freq[(m.rotary.base, m.rotary.dims)]) if m.rotary is not None else (0, None)
        args = (proj, cols, m.heads, m.vdim, m.dim, 1.0 if m.scale_keys else s, s if m.scale_keys else 1.0, rot, freq, *fixed,
                P[p + "a2.weight"] if m.rank else None, P[p + "a2.bias"] if m.rank else None, 1.0 / m.tau, P[p + "norm.weight"] if m.norm_weight else None,
                self.plan.eps, state, meta.state_slots, self.status)
        out = torch.empty(proj.shape[0], P[f"layers.{i}.{side}o.weight"].shape[1], dtype=proj.dtype, device=self.dev)
        if meta.is_prefill:
            t = self._tables(meta)
            fast = not self.plain
            C.linear_prefill(*args, positions, meta.cu_seqlens, meta.ctx_lens, t["chunks"] if fast else None, t["first"] if fast else None, out)
            self.launches += 5
        else:
            C.linear_step(*args, positions, out)
            self.launches += 1
        return out

    # ------------------------------------------------------------------ layers
    def _sequential_layer(self, run, x, h, positions, meta, cache):
        """Updates the fp32 residual ``x`` in place and ``h`` to what the next layer run reads."""
        i = self.runs[run]
        l, P, p, C = self.plan.layers[i], self.store.params, f"layers.{i}.", self.C
        m, eps, f32 = l.mixer, self.plan.eps, torch.float32
        after = f"layers.{self.runs[run + 1]}.norm1" if run + 1 < len(self.runs) else "final_norm"
        proj = self.linear(h, P[p + "in.weight"])
        second = (None, None, None)
        if isinstance(m, Parallel):
            a = self._attention(i, m.left, "left.", proj, positions, meta, cache[0])
            b = self._linear_attention(i, m.right, "right.", proj, positions, meta, cache[1])
            y = self.linear(a, P[p + "left.o.weight"], f32)
            second = (self.linear(b, P[p + "right.o.weight"], f32), P[p + "mix.left.out_norm.weight"], P[p + "mix.right.out_norm.weight"])
        else:
            y = self.linear(self._linear_attention(i, m, "", proj, positions, meta, cache[0]), P[p + "o.weight"], f32)
        C.sandwich(x, y, *second, P[p + "norm1b.weight"], P[(p + "norm2" if l.ff is not None else after) + ".weight"], h, eps)
        self.launches += 1
        if l.ff is not None:
            z = self.linear(h, P[p + "ff_in.weight"])
            gate, up = l.ff_segments()
            w = P[p + "ff_out.weight"]
            act = torch.empty(z.shape[0], w.shape[1], dtype=z.dtype, device=self.dev)
            C.gated_act(z, gate.start, up.start, l.ff.ff, l.ff.act == "relu", act)
            C.sandwich(x, self.linear(act, w, f32), None, None, None, P[p + "norm2b.weight"], P[after + ".weight"], h, eps)
            self.launches += 2

    def _next_norm(self, i):
        return f"layers.{i + 1}.norm1" if i + 1 < self.cfg.num_layers else "final_norm"

    def _layer(self, i, x, h, tokens, positions, meta, cache):
        """Updates the fp32 residual ``x`` in place and ``h`` to the next layer's normed input."""
        l, P, p, C = self.plan.layers[i], self.store.params, f"layers.{i}.", self.C
        T = h.shape[0]
        proj = self.linear(h, P[p + "in.weight"])
        cat = torch.empty(T, l.out_cols, dtype=h.dtype, device=self.dev)
        s = self.in_segs[i]
        ff = (s["mlp.gate"].start, s["mlp.up"].start, l.ff.ff, self.out_segs[i]["mlp.down"].start) if l.ff is not None else (0, 0, 0, 0)
        mix = self._mamba2 if isinstance(l.mixer, Mamba2) else self._latent_attention
        mix(i, proj, cat, ff, meta, cache, positions)
        w_out, delta = P[p + "out.weight"], None
        if self.f32:
            delta = F.linear(cat, w_out)
        elif T <= SMALL_T and w_out.shape[0] % 16 == 0:
            delta = self.linear(cat, w_out, torch.float32)
        else:  # the product's epilogue adds into the residual
            C.gemm(cat, w_out, x, False, False, True, 0, self.status)
            self.launches += 1
        nn = self._next_norm(i)
        gate, sproj = P[p + "side.gate.weight"], P[p + "side.proj.weight"]
        side = (x, None, tokens, gate, sproj, P[p + "side.norm.weight"], P["side.embed.weight"], i, P[nn + ".weight"], P[nn + ".bias"],
                P[nn + ".alpha"], h, self.plan.eps, self.status)
        if T <= FUSED_SIDE_T or self.f32 or sproj.shape[1] % 8 or x.shape[1] % 8 or self.plain:
            C.side_fused(x, delta, *side[2:])
            self.launches += 1
            return
        xb = torch.empty_like(h)
        C.cast_rows(x, delta, xb)
        g = torch.empty(T, gate.shape[0], dtype=h.dtype, device=self.dev)
        C.side_gate(*side, self.linear(xb, gate, torch.float32), g)
        C.side_finish(*side, self.linear(g, sproj, torch.float32))
        self.launches += 3

    @torch.no_grad()
    def forward_hidden(self, tokens, positions, cu_seqlens, meta: Optional[InferMeta] = None, kv_cache=None, replay=None,
                       record=None, max_seqlen: int = 0):
        if meta is None:
            meta, kv_cache = self.scratch_cache(cu_seqlens)
        P = self.store.params
        tokens, positions = tokens.contiguous(), positions.contiguous()
        T, H = tokens.shape[0], self.cfg.hidden_size
        x = torch.empty(T, H, dtype=torch.float32, device=self.dev)
        h = torch.empty(T, H, dtype=self.store.dtype, device=self.dev)
        first = f"layers.{self.runs[0]}.norm1"
        if self.plan.norm == "layer_norm":
            self.C.embed_layer_norm(tokens, P["embed.weight"], P[first + ".weight"], x, h, self.plan.eps, self.status)
        else:
            self.C.embed_norm(tokens, P["embed.weight"], P[first + ".weight"], P[first + ".bias"], P[first + ".alpha"], x, h, self.status)
        self.launches += 1
        for run, i in enumerate(self.runs):
            if self.plan.parallel:
                self._layer(i, x, h, tokens, positions, meta, kv_cache[run])
            else:
                self._sequential_layer(run, x, h, positions, meta, kv_cache[run])
            if self.capture is not None:
                self.capture.append(x.clone())
        return h

    @torch.no_grad()
    def logits(self, hidden_rows):
        return self.linear(hidden_rows.contiguous(), self.store.params["lm_head.weight"], torch.float32)
