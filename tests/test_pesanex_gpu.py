"""Pesanex kernels and models on the GPU against a plain restatement of the equations."""
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import oracle_pesanex as O  # noqa: E402
from pesanex_cases import CASES, RANKS, config, gla, parallel, retention, sharpen, slow  # noqa: E402
from rokivik_cases import feed_all, load, row_errors, tells_apart, tokens_of  # noqa: E402
from test_pesanex import far_key, greedy_gap  # noqa: E402

pytestmark = pytest.mark.gpu
DT = {"fp32": torch.float32, "bf16": torch.bfloat16}


def dev(t, dtype=None):
    return t.to(device="cuda", dtype=dtype or t.dtype).contiguous()


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def ext():
    from miles_b200.ops import _ext

    return _ext.load_hybrid()


def b16(t):
    return t.to(torch.bfloat16).float()


def close(got, want, tol, what=""):
    got, want = got.float().cpu(), want.float()
    err = (got - want).abs().max() / want.abs().max().clamp(min=1e-6)
    assert torch.isfinite(got).all() and err < tol, (what, float(err))


def freqs(base, dims):
    from miles_b200.ops.reference import pair_frequencies

    return pair_frequencies(dims, base, "cuda")


# ------------------------------------------------------------------------------------------------ linear attention
class Linear:
    """Projected rows of one mixer and what they should give."""

    def __init__(self, H, P, N, T, dtype, seed=0, decay=None, rank=0, tau=1.0, shift=2.0, rot=0, norm=False):
        g, gw = torch.Generator().manual_seed(seed), torch.Generator().manual_seed(99)  # (the weights are the same for every sequence)
        r = lambda *s: b16(torch.randn(*s, generator=g))
        self.H, self.P, self.N, self.T, self.dtype, self.rot, self.eps = H, P, N, T, dtype, rot, 1e-5
        parts, self.cols, at = {"v": r(T, H * P), "k": r(T, H * N), "q": r(T, H * N), "g": r(T, H * P), "u": r(T, rank)}, [], 0
        blocks = []
        for n in "vkqgu":  # segments at multiples of 16 columns, as in fused weights
            w = parts[n].shape[1]
            self.cols.append(at if w else -1)
            blocks.append(torch.cat([parts[n], torch.full((T, -w % 16), 1e4)], 1))
            at += blocks[-1].shape[1]
        self.rows = torch.cat(blocks, 1)
        self.s = N ** -0.5
        q, k, v = (parts[n].double().view(T, H, -1) for n in "qkv")
        if rot:
            self.freq = freqs(500.0, rot)
            q, k = (O.rotate_half(x, torch.arange(T), 500.0, rot) for x in (q, k))
        if decay is not None:
            self.decay = torch.tensor(decay, dtype=torch.float64)
            alpha = self.decay.view(1, H, 1).expand(T, H, N)
            self.a2 = self.bias = None
        else:
            self.decay, self.tau = None, tau
            self.a2, self.bias = b16(torch.randn(H * N, rank, generator=gw) / rank ** 0.5), b16(shift + 2 * torch.randn(H * N, generator=gw))
            z = parts["u"].double() @ self.a2.double().T + self.bias.double()
            alpha = torch.exp(torch.nn.functional.logsigmoid(z) / tau).view(T, H, N)
        self.norm = b16(1 + 0.3 * torch.randn(P, generator=gw)) if norm else None
        o = O.recurrence(q * self.s, k, v, alpha)
        self.state = None
        o = O.unit_rms(o, self.eps) * (self.norm.double() if norm else 1.0)
        self.want = (o * O.silu(parts["g"].double().view(T, H, P))).reshape(T, H * P)

    def args(self, rows, state, slots, status):
        fixed = (None, None) if self.decay is None else (dev((self.decay - 1).float()), dev(self.decay.log2().clamp(min=-1e4).float()))
        at = lambda t: None if t is None else dev(t, self.dtype)
        keys = self.decay is not None  # where the scale goes
        return (rows, self.cols, self.H, self.P, self.N, 1.0 if keys else self.s, self.s if keys else 1.0, self.rot, self.freq if self.rot else None, *fixed,
                at(self.a2), at(self.bias), 1.0 / getattr(self, "tau", 1.0), at(self.norm), self.eps, state, slots, status)

    def run(self, cuts, chunked, state, slot, status):
        """The sequence in portions (single tokens through the step kernel), its state in row ``slot``."""
        C, outs, at, k = ext(), [], 0, 0
        while at < self.T:
            n = min(cuts[min(k, len(cuts) - 1)], self.T - at)
            rows, out = dev(self.rows[at:at + n], self.dtype), torch.full((n, self.H * self.P + 5), float("nan"), dtype=self.dtype, device="cuda")
            args = self.args(rows, state, i32([slot]), status)
            pos = torch.arange(at, at + n, dtype=torch.int32, device="cuda")
            if n == 1 and at > 0:
                C.linear_step(*args, pos, out)
            else:
                chunks = [(0, r, min(C.CHUNK, n - r), r // C.CHUNK) for r in range(0, n, C.CHUNK)]
                C.linear_prefill(*args, pos, i32([0, n]), i32([at]), i32(chunks) if chunked else None, i32([0, len(chunks)]) if chunked else None, out)
            assert float(out[:, self.H * self.P:].float().abs().sum()) == 0
            outs.append(out[:, :self.H * self.P])
            at, k = at + n, k + 1
        return torch.cat(outs)


KINDS = {
    "retention": [dict(H=3, P=64, N=32, decay=[0.5, 0.97, 0.9997], rot=32), dict(H=2, P=40, N=24, decay=[1.0, 0.0], rot=8), dict(H=1, P=7, N=10, decay=[0.99], rot=6),
                  dict(H=2, P=128, N=128, decay=[0.95, 0.999], rot=64), dict(H=2, P=136, N=256, decay=[0.9, 0.999], rot=256)],
    "gla": [dict(H=2, P=64, N=64, rank=16, tau=16.0, norm=True), dict(H=3, P=40, N=24, rank=5, tau=16.0, norm=True), dict(H=2, P=128, N=128, rank=64, tau=16.0, shift=6.0, norm=True),
            dict(H=2, P=9, N=33, rank=80, tau=8.0), dict(H=1, P=200, N=112, rank=24, tau=4.0, shift=0.0, norm=True), dict(H=2, P=96, N=48, rank=16, tau=1.0, shift=-6.0),
            dict(H=1, P=32, N=160, rank=16, tau=16.0), dict(H=4, P=48, N=16, rank=8, tau=0.25, shift=0.0)],
}


@pytest.mark.parametrize("spec", [(k, i) for k, v in KINDS.items() for i in range(len(v))], ids=lambda s: f"{s[0]}{s[1]}")
@pytest.mark.parametrize("mode", ["fp32", "bf16", "bf16-chunks"])
def test_linear_attention_in_portions_and_steps(spec, mode):
    d = KINDS[spec[0]][spec[1]]
    dtype = DT[mode.split("-")[0]]
    L = Linear(T=300, dtype=dtype, seed=spec[1], **d)
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    state = torch.full((3, d["H"], d["P"], d["N"]), float("nan"), device="cuda")   # rows of earlier owners are not read
    for cuts in ([300], [128, 2, 3, 1, 129], [256, 1], [5, 1, 1, 1, 1, 2]):
        got = L.run(cuts, mode.endswith("chunks"), state, 2, status).double().cpu()
        e = (got - L.want).abs().view(300, d["H"], -1).amax(-1) / L.want.abs().view(300, d["H"], -1).amax(-1)  # by head: a head whose decay is lost shows
        # (a head whose output is almost nothing is normed up with its rounding: single rows may be far off in bf16)
        assert torch.isfinite(got).all() and e.mean(0).max() < (2e-5 if dtype == torch.float32 else 0.015), (cuts, e.mean(0))
        assert e.max() < 1e-3 if dtype == torch.float32 else e.median(0).values.max() < 0.008, (cuts, e.max(), e.median(0))
    assert int(status) == 0


@pytest.mark.parametrize("lens", [[1, 130, 7, 256, 300], [40] * 300 + [257]])
@pytest.mark.parametrize("kind", list(KINDS))
def test_linear_attention_batch_of_unequal_sequences(lens, kind):
    C, d = ext(), KINDS[kind][0]
    Ls = [Linear(T=n, dtype=torch.bfloat16, seed=i, **d) for i, n in enumerate(lens)]
    cu, chunks, first = [0], [], [0]
    for b, n in enumerate(lens):
        chunks += [(b, cu[-1] + r, min(C.CHUNK, n - r), r // C.CHUNK) for r in range(0, n, C.CHUNK)]
        first.append(len(chunks))
        cu.append(cu[-1] + n)
    B = len(lens)
    state, status = torch.full((B + 1, d["H"], d["P"], d["N"]), float("nan"), device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    rows, out = dev(torch.cat([L.rows for L in Ls]), torch.bfloat16), torch.empty(cu[-1], d["H"] * d["P"], dtype=torch.bfloat16, device="cuda")
    pos = torch.cat([torch.arange(n) for n in lens]).to(torch.int32).cuda()
    C.linear_prefill(*Ls[0].args(rows, state, i32([(b * 7 + 3) % B for b in range(B)]), status), pos, i32(cu), i32([0] * B), i32(chunks), i32(first), out)
    for b, L in enumerate(Ls):
        e = (out[cu[b]:cu[b + 1]].double().cpu() - L.want).abs().amax(1) / L.want.abs().amax(1)
        assert e.mean() < 0.05 and e.median() < 0.01, (b, e.mean(), e.median())
    assert int(status) == 0


def test_state_row_outside_the_cache_is_reported_not_followed():
    L = Linear(T=40, dtype=torch.bfloat16, **KINDS["gla"][0])
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    state = torch.zeros(2, 2, 64, 64, device="cuda")
    for chunked in (False, True):
        status.zero_()
        out = L.run([40], chunked, state, 5, status)
        assert int(status) == 11 and float(state.abs().sum()) == 0 and torch.isfinite(out.float()).all()
    status.zero_()
    ext().linear_step(*L.args(dev(L.rows[:1], torch.bfloat16), state, i32([-1]), status), i32([3]), torch.empty(1, 128, dtype=torch.bfloat16, device="cuda"))
    assert int(status) == 11 and float(state.abs().sum()) == 0


def test_slow_decays_do_not_drift():
    """A state that is only multiplied, 4000 times, by a decay near 1, token by token and in chunks."""
    H, P, N, T = 2, 16, 32, 4000
    L = Linear(H, P, N, 1, torch.bfloat16, decay=[1 - 2.0 ** -12, 1 - 2.0 ** -10])
    zero = L.rows.clone()
    zero[:, L.cols[0]:L.cols[0] + H * P] = 0  # no values: nothing is added
    s0 = torch.randn(1, H, P, N, device="cuda")
    want = s0.double().cpu() * L.decay.view(1, H, 1, 1) ** T
    status, C = torch.zeros(1, dtype=torch.int32, device="cuda"), ext()
    for chunked in (False, True):
        state = s0.clone()
        rows = dev(zero, torch.bfloat16).expand(T, -1).contiguous()
        chunks = [(0, r, min(C.CHUNK, T - r), r // C.CHUNK) for r in range(0, T, C.CHUNK)]
        C.linear_prefill(*L.args(rows, state, i32([0]), status), torch.arange(T, dtype=torch.int32, device="cuda"), i32([0, T]), i32([1]), i32(chunks) if chunked else None,
                         i32([0, len(chunks)]) if chunked else None, torch.empty(T, H * P, dtype=torch.bfloat16, device="cuda"))
        close(state, want, 2e-5, chunked)


# ------------------------------------------------------------------------------------------------ softmax attention
def attention_case(m, lens, news, seed, dtype, page=8):
    """Cache rows of several sequences on shuffled pages, queries of their last ``news`` tokens, and what they should give. One key far
    back takes most of one head's weight in each sequence's last row; a second reference leaves the sink out."""
    g = torch.Generator().manual_seed(seed)
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    width = (G * (d + dv) + 7) // 8 * 8
    pages_per = [(n + page - 1) // page for n in lens]
    perm = (torch.randperm(sum(pages_per), generator=g) + 1).tolist()
    rows = torch.full(((sum(pages_per) + 1) * page, width), 3.0e4)  # (other slots: large, so that reading one shows)
    table = torch.zeros(len(lens), max(pages_per) + 1, dtype=torch.int32)
    sink = b16(torch.randn(H, generator=g) + 1)
    wants, bare, qs, pos, seqs = [], [], [], [], []
    for b, (n, k) in enumerate(zip(lens, news)):
        own = torch.tensor([perm.pop() for _ in range(pages_per[b])])
        table[b, :len(own)] = own.to(torch.int32)
        kk, vv, qq = b16(torch.randn(n, G, d, generator=g)), b16(torch.randn(n, G, dv, generator=g)), b16(torch.randn(k, H, d, generator=g))
        if n > 3:  # far back, on a page border for long sequences
            far = 0 if b % 2 else max(0, (n - 2) // page * page - 1)
            kk[far, -1] = b16(qq[-1, H - 1] / qq[-1, H - 1].norm() * d ** 0.5)
            qq[-1, H - 1] = b16(qq[-1, H - 1] * 3)
        at = torch.arange(n)
        rows[own[at // page] * page + at % page] = torch.cat([kk.view(n, -1), vv.view(n, -1), torch.zeros(n, width - G * (d + dv))], 1)
        s = torch.einsum("ihd,jhd->hij", qq, kk.repeat_interleave(H // G, 1)) * m["scale"]
        p = torch.arange(n - k, n)
        s = s.masked_fill(torch.arange(n)[None] > p[:, None], float("-inf"))
        out = lambda w: torch.einsum("hij,jhd->ihd", w, vv.repeat_interleave(H // G, 1)).reshape(k, -1)
        wants.append(out(O.sink_softmax(s, sink)))
        bare.append(out(torch.softmax(s, -1)))
        qs.append(qq)
        pos += p.tolist()
        seqs += [b] * k
    return dict(rows=dev(rows, dtype), table=dev(table), q=torch.cat(qs), pos=i32(pos), seqs=i32(seqs), page=page, sink=dev(sink, dtype), want=torch.cat(wants), bare=torch.cat(bare))


HEADS = [dict(heads=4, kv_heads=2, dim=64, vdim=64), dict(heads=20, kv_heads=1, dim=32, vdim=48), dict(heads=6, kv_heads=6, dim=128, vdim=128),
         dict(heads=3, kv_heads=1, dim=72, vdim=8), dict(heads=80, kv_heads=2, dim=16, vdim=104), dict(heads=2, kv_heads=1, dim=192, vdim=256)]
ODD_HEADS = [dict(heads=2, kv_heads=1, dim=9, vdim=7), dict(heads=6, kv_heads=3, dim=12, vdim=20), dict(heads=2, kv_heads=2, dim=330, vdim=600)]


def attn_args(m, c, status, sink=True):
    return (m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], c["sink"] if sink else None, c["rows"], c["table"], c["page"], status)


@pytest.mark.parametrize("spec", range(len(HEADS) + len(ODD_HEADS)))
@pytest.mark.parametrize("mode", ["fp32", "bf16"])
def test_decode_attention_over_pages(spec, mode):
    C, m = ext(), dict((HEADS + ODD_HEADS)[spec], scale=0.3)
    lens = [1, 2, 8, 9, 16, 17, 63, 64, 65, 300, 700]
    c = attention_case(m, lens, [1] * len(lens), spec, DT[mode])
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    tol, used = (3e-5 if mode == "fp32" else 0.02), m["heads"] * m["vdim"]
    out = torch.full((len(lens), used + 3), float("nan"), dtype=DT[mode], device="cuda")
    C.attn_plain(*attn_args(m, c, status), dev(c["q"]), c["pos"], None, out)
    close(out[:, :used], c["want"], tol)
    assert (out[:, :used].float().cpu() - c["bare"]).abs().max() > 0.1 * c["want"].abs().max()
    C.attn_plain(*attn_args(m, c, status, sink=False), dev(c["q"]), c["pos"], None, out)
    close(out[:, :used], c["bare"], tol)
    width = c["rows"].shape[1]
    if mode == "bf16" and C.attn_decode_supported(m["heads"], m["kv_heads"], m["dim"], m["vdim"], width):
        for splits in (1, 2, 5, 32, 33, 64):
            for sink in (True, False):
                out.fill_(float("nan"))
                C.attn_decode(*attn_args(m, c, status, sink), dev(c["q"], torch.bfloat16), i32(lens), splits, out)
                close(out[:, :used], c["want"] if sink else c["bare"], tol, splits)
                assert float(out[:, used:].float().abs().sum()) == 0
    else:
        assert mode == "fp32" or spec >= len(HEADS)
    assert int(status) == 0


@pytest.mark.parametrize("spec", range(len(HEADS) + len(ODD_HEADS)))
@pytest.mark.parametrize("mode", ["fp32", "bf16"])
def test_prompt_attention_in_portions(spec, mode):
    C, m = ext(), dict((HEADS + ODD_HEADS)[spec], scale=0.3)
    lens, news = [300, 5, 170, 131, 260, 128, 2], [300, 5, 40, 2, 129, 128, 2]
    c = attention_case(m, lens, news, 20 + spec, DT[mode])
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    used, T = m["heads"] * m["vdim"], sum(news)
    out = torch.empty(T, (used + 31) // 32 * 32, dtype=DT[mode], device="cuda")
    C.attn_plain(*attn_args(m, c, status), dev(c["q"]), c["pos"], c["seqs"], out)
    close(out[:, :used], c["want"], 3e-5 if mode == "fp32" else 0.02)
    if mode == "bf16" and C.attn_prefill_supported(m["kv_heads"], m["dim"], m["vdim"], c["rows"].shape[1]):
        ranges, tiles, at, row = [], [], 0, 0
        for b, (n, k) in enumerate(zip(lens, news)):
            ranges.append((b, 0, at, n))
            tiles += [(row + r, min(128, k - r), at, n - k + r) for r in range(0, k, 128)]
            at, row = at + n, row + k
        pad = 64 if m["dim"] <= 64 else 128
        q = torch.zeros(T, m["heads"], pad)
        q[..., :m["dim"]] = c["q"]
        for sink in (True, False):
            out.fill_(float("nan"))
            C.attn_prefill(*attn_args(m, c, status, sink), dev(q, torch.bfloat16), pad, i32(ranges), at, max(lens), i32(tiles), out)
            close(out[:, :used], c["want"] if sink else c["bare"], 0.03)
    else:
        assert mode == "fp32" or spec >= len(HEADS) - 1
    assert int(status) == 0


def test_page_outside_the_cache_is_reported_not_followed():
    m = dict(HEADS[0], scale=0.2)
    c = attention_case(m, [40], [1], 1, torch.bfloat16)
    c["table"][0, 2] = 10 ** 6
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    out = torch.empty(1, 256, dtype=torch.bfloat16, device="cuda")
    ext().attn_decode(*attn_args(m, c, status), dev(c["q"], torch.bfloat16), i32([40]), 1, out)
    assert int(status) == 9 and torch.isfinite(out.float()).all()
    status.zero_()
    ext().head_rows(dev(torch.randn(1, 64), torch.bfloat16), i32([0]), i32([10 ** 6]), 1e-5, status, [(0, 1, 64, 0, None, False, 1.0, c["rows"], 0, 64, 0, True)])
    assert int(status) == 9


# ------------------------------------------------------------------------------------------------ row-wise kernels
@pytest.mark.parametrize("dims", [(3, 64, 32, 64), (2, 10, 6, 16), (1, 7, 4, 7), (5, 128, 128, 128), (2, 40, 0, 48), (4, 16, 2, 16), (13, 96, 32, 128), (35, 16, 16, 16),
                                  (1, 256, 64, 256), (2, 400, 16, 400)])
@pytest.mark.parametrize("mode", ["fp32", "bf16"])
@pytest.mark.parametrize("T", [50, 600])
def test_rotation_norm_and_layout_of_heads(dims, mode, T):
    H, d, rot, pitch = dims
    dtype, g = DT[mode], torch.Generator().manual_seed(1)
    lead, tail = 16, 8 if pitch % 8 == 0 else 5
    rows, pos = b16(torch.randn(T, lead + 2 * H * d, generator=g)), torch.randint(0, 5000, (T,), generator=g)
    slots = torch.randperm(T + 40, generator=g)[:T]
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    proj, wide = dev(rows, dtype), torch.full((T, 8 + H * pitch), float("nan"), dtype=dtype if T > 100 else torch.float32, device="cuda")
    cache = torch.full((T + 40, H * pitch + tail), float("nan"), dtype=dtype, device="cuda")
    f = freqs(1e4, rot) if rot else None
    ext().head_rows(proj, dev(pos, torch.int32), dev(slots, torch.int32), 1e-3, status,
                    [(lead, H, d, rot, f, True, 1.0, wide, 8, pitch, 0, False), (lead + H * d, H, d, rot, f, True, 0.5, cache, 0, pitch, tail, True)])
    x, y = rows[:, lead:lead + H * d].view(T, H, d), rows[:, lead + H * d:].view(T, H, d)
    tol = 1e-5 if mode == "fp32" else 0.01
    close(wide[:, 8:].view(T, H, pitch)[..., :d], O.unit_rms(O.rotate_half(x, pos, 1e4, rot), 1e-3), 6e-4 if mode == "fp32" else tol)  # (angles in fp32)
    got = cache[slots.cuda()]
    close(got[:, :H * pitch].reshape(T, H, pitch)[..., :d], O.unit_rms(O.rotate_half(y, pos, 1e4, rot), 1e-3) * 0.5, 6e-4 if mode == "fp32" else tol)
    assert float(got[:, H * pitch:].float().abs().sum()) == 0 and float(wide[:, 8:].view(T, H, pitch)[..., d:].float().abs().sum()) == 0
    assert torch.isnan(cache.float()).any(1).sum() == 40 and int(status) == 0


@pytest.mark.parametrize("mode", ["fp32", "bf16"])
@pytest.mark.parametrize("T", [9, 700])
def test_heads_in_place(T, mode):
    rows = b16(torch.randn(T, 96))
    proj, status = dev(rows, DT[mode]), torch.zeros(1, dtype=torch.int32, device="cuda")
    ext().head_rows(proj, i32(list(range(T))), None, 1e-5, status, [(32, 2, 24, 16, freqs(50.0, 16), False, 2.0, proj, 32, 24, 0, False)])
    want = O.rotate_half(rows[:, 32:80].view(T, 2, 24), torch.arange(T), 50.0, 16) * 2
    close(proj[:, 32:80], want.reshape(T, 48), 1e-4 if mode == "fp32" else 0.01)
    proj = proj.float()
    assert torch.equal(proj[:, :32].cpu(), rows[:, :32]) and torch.equal(proj[:, 80:].cpu(), rows[:, 80:])


@pytest.mark.parametrize("T,H", [(1, 64), (3, 50), (200, 256), (9, 2048), (300, 4096), (2, 5000), (160, 8192), (2, 12288), (7, 3)])
@pytest.mark.parametrize("mode", ["fp32", "bf16"])
def test_norms_around_a_sublayer(T, H, mode):
    dtype, g = DT[mode], torch.Generator().manual_seed(T)
    C, eps = ext(), 1e-3
    x, y, z = (torch.randn(T, H, generator=g) * s + 0.5 for s in (2.0, 0.3, 5.0))
    post, nxt, w1, w2 = (b16(1 + 0.3 * torch.randn(H, generator=g)) for _ in range(4))
    h = torch.empty(T, H, dtype=dtype, device="cuda")
    tol = 1e-5 if mode == "fp32" else 0.01
    W = lambda t: dev(t, dtype)
    for two in (False, True):
        gx = dev(x)
        C.sandwich(gx, dev(y), dev(z) if two else None, W(w1) if two else None, W(w2) if two else None, W(post), W(nxt), h, eps)
        yy = (O.unit_rms(y.double(), eps) * w1 + O.unit_rms(z.double(), eps) * w2) / 2 if two else y.double()
        want = x + O.layer_norm(yy, post.double(), eps)
        close(gx, want, 1e-5)
        close(h, O.layer_norm(want, nxt.double(), eps), tol)
    table, toks, status = b16(torch.randn(11, H, generator=g)), torch.randint(0, 11, (T,), generator=g), torch.zeros(1, dtype=torch.int32, device="cuda")
    C.embed_layer_norm(dev(toks, torch.int32), W(table), W(nxt), gx, h, eps, status)
    close(gx, table[toks], 1e-6)
    close(h, O.layer_norm(table[toks].double(), nxt.double(), eps), tol)
    assert int(status) == 0
    C.embed_layer_norm(i32([11] * T), W(table), W(nxt), gx, h, eps, status)
    assert int(status) == 10


@pytest.mark.parametrize("ff,ldo", [(48, 64), (37, 64), (7, 32), (256, 256)])
@pytest.mark.parametrize("mode", ["fp32", "bf16"])
@pytest.mark.parametrize("relu", [True, False])
def test_gated_activation(ff, ldo, mode, relu):
    up = (ff + 15) // 16 * 16
    rows = b16(torch.randn(33, up + ff + 3))
    out = torch.full((33, ldo), float("nan"), dtype=DT[mode], device="cuda")
    ext().gated_act(dev(rows, DT[mode]), 0, up, ff, relu, out)
    g, u = rows[:, :ff], rows[:, up:up + ff]
    close(out[:, :ff], (torch.clamp(g, min=0) if relu else O.silu(g)) * u, 1e-5 if mode == "fp32" else 0.01)
    assert float(out[:, ff:].float().abs().sum()) == 0


# ------------------------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module", params=[(k, m) for k in CASES for m in DT], ids=lambda p: "-".join(p))
def served(request, tmp_path_factory):
    name, mode = request.param
    cfg = CASES[name]
    W = O.random_weights(cfg, seed=3, dtype=torch.float32, rank=RANKS.get(name))
    eng = load(cfg, W, tmp_path_factory.mktemp("m"), "cuda", DT[mode], num_pages=200, max_seq_len=512)
    yield cfg, W, eng, DT[mode]
    eng.model.check_status()


def agree(got, want, dtype):
    """Logits agree up to rounding; a row in which some head's output is almost nothing is normed up with its rounding, so that single
    rows are held loosely."""
    e = row_errors(got, want)
    return bool(e.mean() < 2e-5 and e.max() < 1e-3) if dtype == torch.float32 else bool(e.mean() < 0.04 and e.max() < 0.6)


def test_whole_prompt_single_tokens_and_portions(served):
    cfg, W, eng, dtype = served
    toks = tokens_of(301, cfg["vocab"], 1)
    want = O.model(cfg, W, toks)
    for cuts in ([301], [128, 2, 3, 100, 1], [7], [290, 1]):
        assert agree(feed_all(eng, "a", toks, cuts), want, dtype), cuts
    assert agree(feed_all(eng, "a", toks[:40], [2, 1]), want[:40], dtype)


def test_layers_one_by_one(served):
    cfg, W, eng, dtype = served
    toks, ref = tokens_of(40, cfg["vocab"], 5), []
    O.model(cfg, W, toks, ref)
    eng.model.capture = got = []
    eng.model.forward_hidden(i32(toks), torch.arange(40, dtype=torch.int32, device="cuda"), i32([0, 40]))
    eng.model.capture = None
    assert len(got) == len(ref)
    for i, (a, b) in enumerate(zip(got, ref)):
        e = (a.cpu() - b).pow(2).mean(-1).sqrt() / b.pow(2).mean().sqrt()
        assert e.mean() < (2e-5 if dtype == torch.float32 else 0.04), (i, e.mean())


def test_unequal_batch_reused_rows_and_decode_batch(served):
    cfg, W, eng, dtype = served
    free = eng.pool.num_free
    for rnd in range(2):  # the second round gets pages and state rows that the first one gave back
        seqs = {f"{rnd}-{n}": tokens_of(n, cfg["vocab"], n + rnd) for n in (5, 140, 33, 70)}
        want = {k: O.model(cfg, W, t) for k, t in seqs.items()}
        rows = []
        got = eng.feed([(k, t[:-3], [len(t) - 4]) for k, t in seqs.items()])
        for (k, t), g in zip(seqs.items(), got):
            rows.append((g.cpu(), want[k][len(t) - 4:len(t) - 3]))
        for j in (3, 2, 1):
            order = list(seqs)[::-1] if j == 2 else list(seqs)
            got = eng.feed([(k, [seqs[k][-j]], [0]) for k in order])
            for k, g in zip(order, got):
                rows.append((g.cpu(), want[k][len(seqs[k]) - j][None]))
        assert agree(torch.cat([a for a, _ in rows]), torch.cat([b for _, b in rows]), dtype)
        for k in seqs:
            eng.end_feed(k)
    assert eng.pool.num_free == free


def test_greedy_generation_through_the_scheduler(served):
    """Captured decode graphs, one step in flight, more requests than rows, portions of prompts, pages running dry."""
    cfg, W, eng0, dtype = served
    import miles_b200.engine as E

    eng = E.Engine(eng0.model, max_running=3, num_pages=34, page_size=8, max_seq_len=160, max_prefill_tokens=50)
    prompts = [tokens_of(n, cfg["vocab"], n) for n in (90, 5, 64, 17, 33)]
    outs = eng.generate(prompts, E.SamplingParams(temperature=0.0, max_new_tokens=60))
    for p, o in zip(prompts, outs):
        assert len(o["output_ids"]) == 60 and greedy_gap(cfg, W, p, o["output_ids"]) < (1e-3 if dtype == torch.float32 else 0.3)
    assert eng.pool.num_free == 33 and len(eng.slots_free) == 3


def test_plain_and_tensor_core_kernels_agree(tmp_path):
    cfg = CASES["tiles"]
    W = O.random_weights(cfg, seed=4, dtype=torch.float32, rank=RANKS["tiles"])
    eng = load(cfg, W, tmp_path, "cuda", torch.bfloat16, num_pages=200, max_seq_len=512)
    toks = tokens_of(280, cfg["vocab"], 2)
    fast = feed_all(eng, "a", toks, [260, 1])
    eng.model.plain, eng.use_cuda_graph = True, False
    assert agree(feed_all(eng, "b", toks, [260, 1]), fast, torch.bfloat16)


@pytest.mark.parametrize("mode", list(DT))
@pytest.mark.parametrize("back", [1, 15, 16, 17, 127, 128, 129, 299])
def test_one_far_key_decides_a_row(tmp_path, mode, back):
    cfg = config([parallel(scale=12.0, dims=2, ff=0)])
    W = O.random_weights(cfg, seed=1, dtype=torch.float32)
    eng = load(cfg, W, tmp_path, "cuda", DT[mode], num_pages=100, max_seq_len=400, page_size=16)
    toks, other = far_key(cfg, W, 300, back)
    want, wrong = O.model(cfg, W, toks), O.model(cfg, W, other)
    for cuts in ([300], [299, 1], [300 - back, 2], [128]):
        got = feed_all(eng, "a", toks, cuts)
        assert row_errors(got, want).mean() < (5e-5 if mode == "fp32" else 0.03), cuts
        assert tells_apart(got[299:], want[299:], wrong[299:])


@pytest.mark.parametrize("mode", list(DT))
def test_sharp_attention_first_tokens_and_sinks(tmp_path, mode):
    cfg = config([parallel(heads=8, kv_heads=2, dim=32, vdim=32, dims=16, scale=1.0)])
    cfg, W = sharpen(cfg, O.random_weights(cfg, seed=5, dtype=torch.float32), 2.0)
    eng = load(cfg, W, tmp_path, "cuda", DT[mode], num_pages=100, max_seq_len=400, page_size=16)
    toks = tokens_of(200, cfg["vocab"], 4)
    want, bare = O.model(cfg, W, toks), O.model(cfg, dict(W, **{"l0.mix.left.sink": torch.full((8,), -50.0)}), toks)
    for cuts in ([200], [2], [70, 1]):
        got = feed_all(eng, "a", toks, cuts)
        assert row_errors(got, want).mean() < (5e-5 if mode == "fp32" else 0.03), cuts
        assert tells_apart(got, want, bare) and tells_apart(got[:3], want[:3], bare[:3])


def test_long_decoding_keeps_the_state_exact(tmp_path):
    cfg = config([gla(heads=4, dim=32, vdim=64), parallel(), retention(heads=2, decay=[0.9999, 1.0])], loop=(0, 2, 2))
    W = slow(O.random_weights(cfg, seed=8, dtype=torch.float32))
    for mode in DT:
        eng = load(cfg, W, tmp_path / mode, "cuda", DT[mode], num_pages=200, max_seq_len=900)
        toks = tokens_of(800, cfg["vocab"], 1)
        assert agree(feed_all(eng, "a", toks, [2, 1]), O.model(cfg, W, toks), DT[mode])


def test_wide_decode_batch_takes_the_tensor_core_products(tmp_path):
    """More rows than the few-row kernels serve: products run in their prompt form inside a decode step."""
    cfg = CASES["tiles"]
    W = O.random_weights(cfg, seed=4, dtype=torch.float32, rank=RANKS["tiles"])
    eng = load(cfg, W, tmp_path, "cuda", torch.bfloat16, num_pages=1500, max_seq_len=64, max_running=300, page_size=8)
    seqs = {str(k): tokens_of(9 + k % 7, cfg["vocab"], k) for k in range(290)}
    eng.feed([(k, t[:-1], []) for k, t in seqs.items()])
    got = eng.feed([(k, t[-1:], [0]) for k, t in seqs.items()])
    pick = (0, 1, 137, 288, 289)
    assert agree(torch.cat([got[k] for k in pick]).cpu(), torch.cat([O.model(cfg, W, seqs[str(k)])[-1:] for k in pick]), torch.bfloat16)
