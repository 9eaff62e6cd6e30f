"""PyTorch execution of models with a layer plan (``models/layer_plan.py``): the CPU configuration of the engine and its
scheduler, and the common parts of the sm_100a path (``b200_hybrid.py``).

Model protocol as in ``torch_impl``: packed tokens with ``cu_seqlens``, an ``InferMeta`` that says where every sequence's
cache is, ``forward_hidden`` -> final-normed hidden rows, ``logits``. A pass brings, for every sequence, the tokens that
follow ``meta.ctx_lens`` cached ones: whole prompts, portions of prompts and single tokens are the same operation.
Without ``meta`` (scoring) a temporary cache is used.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn.functional as F

from ..ops import reference as R
from .cache_layout import cache_layout
from .config import ModelConfig
from .layer_plan import Mamba2, Parallel
from .params import ParamStore
from .torch_impl import InferMeta


class TorchHybrid:
    def __init__(self, cfg: ModelConfig, store: ParamStore):
        assert cfg.plan is not None and store.pp_size == 1 and store.tp_size == 1, "planned layers run on one rank"
        self.cfg, self.plan, self.store = cfg, cfg.plan, store
        self.dev = store.device
        self.in_segs = [{s.name: s for s in l.in_segments()} for l in cfg.plan.layers]
        self.out_segs = [{s.name: s for s in l.out_segments()} if l.parallel else {} for l in cfg.plan.layers]
        self.runs = cfg.plan.runs()
        self.capture: Optional[list] = None   # a list: receives the residual stream after every layer run

    # ------------------------------------------------------------------ pieces
    def linear(self, x, w):
        return F.linear(x, w)

    def _norm(self, x, name):
        P = self.store.params
        if self.plan.norm == "layer_norm":
            return R.layer_norm(x, P[name + ".weight"], self.plan.eps).to(self.store.dtype)
        return R.dynamic_tanh(x, P[name + ".weight"], P[name + ".bias"], P[name + ".alpha"]).to(self.store.dtype)

    def _part(self, i, proj, name):
        s = self.in_segs[i]["mix." + name]
        return proj[:, s.start:s.start + s.size]

    def _sequences(self, meta: InferMeta, n_rows: int):
        """(first row, rows, cached tokens, pages, state slot) of every sequence of the pass."""
        slots = meta.state_slots.tolist()
        if meta.is_prefill:
            cu = meta.cu_seqlens.tolist()
            ctx = meta.ctx_lens.tolist()
            return [(cu[b], cu[b + 1] - cu[b], ctx[b], meta.block_table[b].long(), slots[b]) for b in range(len(ctx))]
        lens = meta.seq_lens.tolist()
        return [(b, 1, lens[b] - 1, meta.block_table[b].long(), slots[b]) for b in range(n_rows)]

    def _mamba2(self, i, proj, meta, cache):
        m, P, p = self.plan.layers[i].mixer, self.store.params, f"layers.{i}.mix."
        conv, ssm = cache
        outs = []
        for r0, n, ctx, _, slot in self._sequences(meta, proj.shape[0]):
            z, xbc, dt = proj[r0:r0 + n].split([m.inner, m.channels, m.heads], -1)
            # the ring holds the inputs of positions ctx - taps .. ctx - 1, position p in row p % taps
            old = [conv[slot, q % m.conv] if q >= 0 else torch.zeros_like(conv[slot, 0]) for q in range(ctx - m.conv + 1, ctx)]
            seq = torch.cat([torch.stack(old).to(xbc.dtype), xbc]) if old else xbc
            for q in range(max(0, n - m.conv), n):
                conv[slot, (ctx + q) % m.conv] = xbc[q].to(conv.dtype)
            act = R.causal_conv_silu(seq, P[p + "conv.weight"], P[p + "conv.bias"])
            x, B, C = act.float().split([m.inner, m.groups * m.state, m.groups * m.state], -1)
            S = ssm[slot].clone() if ctx > 0 else torch.zeros_like(ssm[slot])
            y, S = R.state_space_scan(x.view(n, m.heads, m.vdim), B.view(n, m.groups, m.state), C.view(n, m.groups, m.state),
                                      dt.float() + P[p + "dt_bias"].float(), P[p + "A_log"].float(), P[p + "D"].float(), S)
            ssm[slot] = S
            g = y.reshape(n, m.inner) * F.silu(z.float())
            g = R.unit_rms(g.view(n, m.norm_groups, -1), self.plan.eps).view(n, m.inner) * P[p + "norm.weight"].float()
            outs.append(g.to(proj.dtype))
        return torch.cat(outs)

    def _latent_attention(self, i, proj, positions, meta, cache):
        m, P, p = self.plan.layers[i].mixer, self.store.params, f"layers.{i}.mix."
        eps, rows = self.plan.eps, cache[0]
        part = lambda name: self._part(i, proj, name)
        cq = (R.unit_rms(part("dq").float(), eps) * P[p + "q_norm.weight"].float()).to(proj.dtype)
        q = self.linear(cq, P[p + "uq.weight"]).view(-1, m.heads, m.dim + m.rot_dim)
        qn, qr = q[..., :m.dim], R.rotate_pairs(q[..., m.dim:], positions, m.rotary.base)
        if m.kv_from is None:
            t = part("dkv").float()
            c = R.unit_rms(t[:, :m.kv_rank], eps) * P[p + "kv_norm.weight"].float()
            new = torch.cat([c, R.rotate_pairs(t[:, None, m.kv_rank:], positions, m.rotary.base)[:, 0]], 1)
            rows[meta.slot_mapping.long(), :new.shape[1]] = new.to(rows.dtype)
        ps, outs = meta.page_size, []
        wk, wv = P[p + "ukv.weight"].split([m.heads * m.dim, m.heads * m.vdim])
        for r0, n, ctx, pages, _ in self._sequences(meta, proj.shape[0]):
            lo = max(0, ctx - m.window + 1) if m.window else 0
            at = torch.arange(lo, ctx + n, device=proj.device)
            kv = rows[pages[at // ps] * ps + at % ps].to(proj.dtype)
            c, kr = kv[:, :m.kv_rank], kv[:, m.kv_rank:m.kv_rank + m.rot_dim]
            k = self.linear(c, wk).view(-1, m.heads, m.dim)
            v = self.linear(c, wv).view(-1, m.heads, m.vdim)
            s = (torch.einsum("ihd,jhd->hij", qn[r0:r0 + n].float(), k.float())
                 + torch.einsum("ihd,jd->hij", qr[r0:r0 + n].float(), kr.float())) * m.scale
            back = (torch.arange(ctx, ctx + n, device=proj.device)[:, None] - at[None, :])
            seen = (back >= 0) & ((back < m.window) if m.window else (back >= 0))
            a = torch.softmax(s.masked_fill(~seen, float("-inf")), -1)
            outs.append(torch.einsum("hij,jhd->ihd", a, v.float()).reshape(n, -1).to(proj.dtype))
        return torch.cat(outs)

    def _attention(self, i, m, pre, proj, positions, meta, rows):
        """Softmax attention over cached key / value heads; ``pre``: name of the side the mixer is on."""
        T, dt = proj.shape[0], proj.dtype
        sink = self.store.params[f"layers.{i}.mix.{pre}sink"].float() if m.sink else None

        def turned(x):
            x = R.rotate_halves(x, positions, m.rotary.base, m.rotary.dims) if m.rotary is not None else x.float()
            return (R.unit_rms(x, self.plan.eps) if m.unit_qk else x).to(dt)

        q = turned(self._part(i, proj, pre + "q").reshape(T, m.heads, m.dim))
        k = turned(self._part(i, proj, pre + "k").reshape(T, m.kv_heads, m.dim))
        new = torch.cat([k.reshape(T, -1), self._part(i, proj, pre + "v")], 1)
        rows[meta.slot_mapping.long(), :new.shape[1]] = new.to(rows.dtype)
        ps, outs, rep, nk = meta.page_size, [], m.heads // m.kv_heads, m.kv_heads * m.dim
        for r0, n, ctx, pages, _ in self._sequences(meta, T):
            at = torch.arange(ctx + n, device=proj.device)
            kv = rows[pages[at // ps] * ps + at % ps].float()
            kk = kv[:, :nk].view(-1, m.kv_heads, m.dim).repeat_interleave(rep, 1)
            vv = kv[:, nk:nk + m.kv_heads * m.vdim].view(-1, m.kv_heads, m.vdim).repeat_interleave(rep, 1)
            s = torch.einsum("ihd,jhd->hij", q[r0:r0 + n].float(), kk) * m.scale
            s = s.masked_fill(at[None, :] > torch.arange(ctx, ctx + n, device=proj.device)[:, None], float("-inf"))
            outs.append(torch.einsum("hij,jhd->ihd", R.sink_softmax(s, sink), vv).reshape(n, -1).to(dt))
        return torch.cat(outs)

    def _linear_attention(self, i, m, pre, proj, positions, meta, states):
        P, p, T = self.store.params, f"layers.{i}.mix.{pre}", proj.shape[0]
        q, k, v, g = (self._part(i, proj, pre + n) for n in ("q", "k", "v", "g"))
        q, k, v = q.reshape(T, m.heads, m.dim).float(), k.reshape(T, m.heads, m.dim).float(), v.reshape(T, m.heads, m.vdim).float()
        if m.rotary is not None:
            q, k = (R.rotate_halves(x, positions, m.rotary.base, m.rotary.dims) for x in (q, k))
        if m.scale_keys:
            k = k * m.dim ** -0.5
        else:
            q = q * m.dim ** -0.5
        if m.rank:
            z = F.linear(self._part(i, proj, pre + "a1").float(), P[p + "a2.weight"].float()) + P[p + "a2.bias"].float()
            decay = (F.logsigmoid(z) / m.tau).view(T, m.heads, m.dim)
        else:
            decay = torch.tensor(m.decay, dtype=torch.float64, device=proj.device).log().float().view(1, -1, 1)
        outs = []
        for r0, n, ctx, _, slot in self._sequences(meta, T):
            S = states[slot].clone() if ctx > 0 else torch.zeros_like(states[slot])
            at = slice(r0, r0 + n)
            o, states[slot] = R.linear_attention_scan(q[at], k[at], v[at], decay[at] if m.rank else decay, S)
            outs.append(o)
        o = R.unit_rms(torch.cat(outs), self.plan.eps)
        if m.norm_weight:
            o = o * P[p + "norm.weight"].float()
        return (o.reshape(T, -1) * F.silu(g.float())).to(proj.dtype)

    def _project_out(self, w, y):
        """A product whose matrix has padding columns."""
        return self.linear(F.pad(y, (0, w.shape[1] - y.shape[1])), w).float()

    def _sequential_layer(self, i, x, positions, meta, cache):
        """``x + norm(mixer(norm(x)))``, then the same around the feed-forward."""
        l, P, p = self.plan.layers[i], self.store.params, f"layers.{i}."
        m, eps = l.mixer, self.plan.eps
        proj = self.linear(self._norm(x, p + "norm1"), P[p + "in.weight"])
        if isinstance(m, Parallel):
            a = self._attention(i, m.left, "left.", proj, positions, meta, cache[0])
            b = self._linear_attention(i, m.right, "right.", proj, positions, meta, cache[1])
            y = sum(R.unit_rms(self._project_out(P[p + f"{s}.o.weight"], o), eps) * P[p + f"mix.{s}.out_norm.weight"].float()
                    for s, o in (("left", a), ("right", b))) / 2
        else:
            y = self._project_out(P[p + "o.weight"], self._linear_attention(i, m, "", proj, positions, meta, cache[0]))
        x = x + R.layer_norm(y, P[p + "norm1b.weight"], eps)
        if l.ff is not None:
            s = {s.name: s for s in l.ff_segments()}
            z = self.linear(self._norm(x, p + "norm2"), P[p + "ff_in.weight"])
            g, u = (z[:, s[n].start:s[n].start + l.ff.ff] for n in ("mlp.gate", "mlp.up"))
            y = self._project_out(P[p + "ff_out.weight"], (F.relu(g) if l.ff.act == "relu" else F.silu(g)) * u)
            x = x + R.layer_norm(y, P[p + "norm2b.weight"], eps)
        return x

    def _layer(self, i, x, h, tokens, positions, meta, cache):
        l, P, p = self.plan.layers[i], self.store.params, f"layers.{i}."
        proj = self.linear(h, P[p + "in.weight"])
        if isinstance(l.mixer, Mamba2):
            mixed = self._mamba2(i, proj[:, :self.in_segs[i]["mix.in"].size], meta, cache)
        else:
            mixed = self._latent_attention(i, proj, positions, meta, cache)
        cat = h.new_zeros(h.shape[0], l.out_cols)
        cat[:, :mixed.shape[1]] = mixed
        if l.ff is not None:
            g, u, d = self.in_segs[i]["mlp.gate"], self.in_segs[i]["mlp.up"], self.out_segs[i]["mlp.down"]
            cat[:, d.start:d.start + d.size] = F.silu(proj[:, g.start:g.start + g.size]) * proj[:, u.start:u.start + u.size]
        x = x + self.linear(cat, P[p + "out.weight"]).float()
        sd = self.plan.token_side
        e = P["side.embed.weight"][tokens.long(), i * sd:(i + 1) * sd]
        g = F.gelu(self.linear(x.to(h.dtype), P[p + "side.gate.weight"]), approximate="tanh") * e
        y = self.linear(g, P[p + "side.proj.weight"]).float()
        return x + R.unit_rms(y, self.plan.eps) * P[p + "side.norm.weight"].float()

    # ------------------------------------------------------------------ whole passes
    def scratch_cache(self, cu_seqlens, page_size: int = 64):
        """An ``InferMeta`` and a cache for a pass over whole sequences that keeps nothing."""
        cu = [int(v) for v in cu_seqlens.tolist()]
        lens = [b - a for a, b in zip(cu[:-1], cu[1:])]
        pages = [(n + page_size - 1) // page_size for n in lens]
        table = torch.zeros(len(lens), max(pages), dtype=torch.int32)
        slots, at = [], 0
        for b, (n, k) in enumerate(zip(lens, pages)):
            table[b, :k] = torch.arange(at, at + k)
            slots.append(torch.arange(n) + at * page_size)
            at += k
        i32 = dict(dtype=torch.int32, device=self.dev)
        meta = InferMeta(True, cu_seqlens, max(lens), torch.cat(slots).to(**i32), table.to(self.dev), None, page_size, cu,
                         ctx_lens=torch.zeros(len(lens), **i32), ctx_list=[0] * len(lens), state_slots=torch.arange(len(lens), **i32))
        return meta, cache_layout(self.cfg, self.store.dtype).allocate(at * page_size, len(lens), self.dev)

    def forward_hidden(self, tokens, positions, cu_seqlens, meta: Optional[InferMeta] = None, kv_cache=None, replay=None,
                       record=None, max_seqlen: int = 0):
        if meta is None:
            meta, kv_cache = self.scratch_cache(cu_seqlens)
        P = self.store.params
        x = P["embed.weight"][tokens.long()].float()
        for i, cache in zip(self.runs, kv_cache):
            if self.plan.parallel:
                x = self._layer(i, x, self._norm(x, f"layers.{i}.norm1"), tokens, positions, meta, cache)
            else:
                x = self._sequential_layer(i, x, positions, meta, cache)
            if self.capture is not None:
                self.capture.append(x.clone())
        return self._norm(x, "final_norm")

    def logits(self, hidden_rows):
        return self.linear(hidden_rows, self.store.params["lm_head.weight"]).float()

    @torch.no_grad()
    def forward_logprobs(self, tokens, positions, cu_seqlens, row_index, targets, inv_temp, replay=None, record=None,
                         max_seqlen: int = 0, **_):
        """Log-probs / entropy of ``targets`` predicted at packed rows ``row_index`` (scoring; there is no backward)."""
        h = self.forward_hidden(tokens, positions, cu_seqlens, max_seqlen=max_seqlen)[row_index.long()]
        lps, ents = [], []
        for a in range(0, h.shape[0], 2048):
            lp, ent = R.logprob_entropy(self.logits(h[a:a + 2048]), targets[a:a + 2048], inv_temp)
            lps.append(lp)
            ents.append(ent)
        return torch.cat(lps), torch.cat(ents)

    def forward_backward(self, *a, **k):
        raise NotImplementedError(f"{self.plan.design} is served, not trained: its mixers have no backward pass here")
