"""Rokivik kernels and models on the GPU against a plain fp32 restatement of the equations."""
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import oracle_rokivik as O  # noqa: E402
from rokivik_cases import CASES, config, feed_all, latent, load, mamba, near, rel, row_errors, sharpen, tells_apart, tokens_of, with_window  # noqa: E402

pytestmark = pytest.mark.gpu
DT = {"fp32": torch.float32, "bf16": torch.bfloat16}


def dev(t, dtype=None):
    return t.to(device="cuda", dtype=dtype or t.dtype).contiguous()


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def ext():
    from miles_b200.ops import _ext

    return _ext.load_hybrid()


def close(got, want, tol, what=""):
    got, want = got.float().cpu(), want.float()
    err = (got - want).abs().max() / want.abs().max().clamp(min=1e-6)
    assert torch.isfinite(got).all() and err < tol, (what, float(err))


# ------------------------------------------------------------------------------------------------ Mamba-2
def mamba_inputs(H, P, N, G, taps, T, seed, dtype, slow=False):
    g = torch.Generator().manual_seed(seed)
    inner, ch = H * P, H * P + 2 * G * N
    r = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).float()
    d = dict(z=r(T, inner), xbc=r(T, ch), dt=r(T, H), w=r(ch, taps) * 0.5, b=r(ch) * 0.2, bias=r(H) - 2, A=r(H) * 0.7 - (5.0 if slow else 0.0), D=r(H))
    d = {k: v.to(torch.bfloat16).float() for k, v in d.items()}
    pad = torch.zeros(T, 16 - (inner + ch + H) % 16)
    d["proj"] = dev(torch.cat([d["z"], d["xbc"], d["dt"], pad], 1), dtype)
    d["weights"] = [dev(d[k], dtype) for k in ("w", "b", "bias", "A", "D")]
    return d


def mamba_want(d, H, P, N, G):
    act = O.silu(O.causal_conv(d["xbc"], d["w"], d["b"]))
    x, B, C = act.split([H * P, G * N, G * N], 1)
    T = x.shape[0]
    return O.state_space(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), O.softplus(d["dt"] + d["bias"]), d["A"], d["D"]).reshape(T, -1)


def run_portions(d, H, P, N, G, taps, cuts, dtype, chunked, ring, state, slot, status):
    """The sequence in portions (single tokens through the step kernel), its state in row ``slot``."""
    C, outs, at, k, T = ext(), [], 0, 0, d["proj"].shape[0]
    while at < T:
        n = min(cuts[min(k, len(cuts) - 1)], T - at)
        proj = d["proj"][at:at + n].contiguous()
        y = torch.empty(n, H * P, dtype=dtype, device="cuda")
        args = (proj, H, P, N, G, *d["weights"], ring, state, i32([slot]), status)
        if n == 1 and at > 0:
            C.mamba_step(*args, i32([at]), y)
        else:
            conv = [(0, r, min(32, n - r), 0) for r in range(0, n, 32)]
            chunks = [(0, r, min(C.CHUNK, n - r), r // C.CHUNK) for r in range(0, n, C.CHUNK)]
            C.mamba_prefill(*args, i32([0, n]), i32([at]), i32(conv), i32(chunks) if chunked else None, i32([0, len(chunks)]) if chunked else None, y)
        outs.append(y)
        at, k = at + n, k + 1
    return torch.cat(outs)


@pytest.mark.parametrize("dims", [(4, 64, 128, 2, 4), (3, 40, 24, 1, 3), (6, 16, 48, 3, 2), (2, 9, 33, 2, 6), (2, 128, 64, 1, 4), (8, 32, 256, 2, 4), (2, 96, 16, 1, 1),
                                  (12, 64, 128, 1, 4)])
@pytest.mark.parametrize("mode", ["fp32", "bf16", "bf16-chunks"])
def test_recurrence_in_portions_and_steps(dims, mode):
    H, P, N, G, taps = dims
    dtype = DT[mode.split("-")[0]]
    d = mamba_inputs(H, P, N, G, taps, 300, 1, dtype, slow=True)
    want = mamba_want(d, H, P, N, G)
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    ring = torch.full((3, taps, H * P + 2 * G * N), float("nan"), dtype=dtype, device="cuda")   # rows of earlier owners are not read
    state = torch.full((3, H, P, N), float("nan"), device="cuda")
    for cuts in ([300], [128, 2, 3, 1, 129], [256, 1], [5, 1, 1, 1, 1, 2]):
        got = run_portions(d, H, P, N, G, taps, cuts, dtype, mode.endswith("chunks"), ring, state, 2, status)
        close(got, want, 2e-5 if dtype == torch.float32 else 0.02, cuts)
    assert int(status) == 0


@pytest.mark.parametrize("lens", [[1, 130, 7, 256, 300], [40] * 500 + [257]])
@pytest.mark.parametrize("dims", [(4, 64, 64, 2, 4), (24, 32, 32, 3, 4)])
def test_recurrence_batch_of_unequal_sequences(lens, dims):
    """(the long batch also gives every block of the chunked form several heads of a group)"""
    H, P, N, G, taps = dims
    C = ext()
    ds = [mamba_inputs(H, P, N, G, taps, n, 10 + i, torch.bfloat16) for i, n in enumerate(lens)]
    proj = torch.cat([d["proj"] for d in ds])
    w = ds[0]["weights"]
    for d in ds:
        d["w"], d["b"], d["bias"], d["A"], d["D"] = (t.float().cpu() for t in w)
    cu = [0]
    conv, chunks, first = [], [], [0]
    for b, n in enumerate(lens):
        conv += [(b, cu[-1] + r, min(32, n - r), 0) for r in range(0, n, 32)]
        chunks += [(b, cu[-1] + r, min(C.CHUNK, n - r), r // C.CHUNK) for r in range(0, n, C.CHUNK)]
        first.append(len(chunks))
        cu.append(cu[-1] + n)
    B = len(lens)
    ring = torch.zeros(B + 1, taps, H * P + 2 * G * N, dtype=torch.bfloat16, device="cuda")
    state = torch.zeros(B + 1, H, P, N, device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    y = torch.empty(cu[-1], H * P, dtype=torch.bfloat16, device="cuda")
    C.mamba_prefill(proj, H, P, N, G, *w, ring, state, i32([(b * 7 + 3) % B for b in range(B)]), status, i32(cu), i32([0] * B), i32(conv), i32(chunks), i32(first), y)
    for b, d in enumerate(ds):
        if b < 4 or b > B - 3:
            close(y[cu[b]:cu[b + 1]], mamba_want(d, H, P, N, G), 0.02, lens[b])
    assert int(status) == 0


def test_state_row_outside_the_cache_is_reported_not_followed():
    H, P, N, G = 2, 16, 16, 1
    d = mamba_inputs(H, P, N, G, 4, 1, 1, torch.bfloat16)
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    ring = torch.zeros(2, 4, H * P + 2 * N, dtype=torch.bfloat16, device="cuda")
    state = torch.zeros(2, H, P, N, device="cuda")
    ext().mamba_step(d["proj"], H, P, N, G, *d["weights"], ring, state, i32([7]), status, i32([3]), torch.empty(1, H * P, dtype=torch.bfloat16, device="cuda"))
    assert int(status) == 11 and float(state.abs().sum()) == 0
    d = mamba_inputs(H, P, N, G, 4, 40, 1, torch.bfloat16)
    for chunked in (False, True):
        status.zero_()
        y = run_portions(d, H, P, N, G, 4, [40], torch.bfloat16, chunked, ring, state, 2, status)
        assert int(status) == 11 and float(state.abs().sum()) == 0 and torch.isfinite(y.float()).all()


@pytest.mark.parametrize("inner,groups", [(64, 1), (96, 3), (512, 8), (130, 13), (4096, 2), (21, 7)])
@pytest.mark.parametrize("mode", ["fp32", "bf16"])
@pytest.mark.parametrize("rows", [5, 200])
def test_gated_group_norm_and_feed_forward_tail(inner, groups, mode, rows):
    dtype, g = DT[mode], torch.Generator().manual_seed(0)
    ff, gate = 40, (inner + 15) // 16 * 16
    up, down = gate + 48, (inner + 31) // 32 * 32
    y, proj, w = (torch.randn(*s, generator=g).to(torch.bfloat16).float() for s in ((rows, inner), (rows, up + 48), (inner,)))
    cat = torch.full((rows, down + 64), float("nan"), dtype=dtype, device="cuda")
    ext().mamba_tail(dev(y, dtype), dev(w, dtype), groups, 1e-5, dev(proj, dtype), cat, gate, up, ff, down)
    v = (y * O.silu(proj[:, :inner])).view(rows, groups, -1)
    close(cat[:, :inner], O.unit_rms(v, 1e-5).view(rows, inner) * w, 1e-5 if mode == "fp32" else 0.01)
    close(cat[:, down:down + ff], O.silu(proj[:, gate:gate + ff]) * proj[:, up:up + ff], 1e-5 if mode == "fp32" else 0.01)
    assert float(cat[:, inner:down].float().abs().sum() + cat[:, down + ff:].float().abs().sum()) == 0  # columns nobody owns are zeros


# ------------------------------------------------------------------------------------------------ per-layer token input
@pytest.mark.parametrize("T,H,sd", [(1, 64, 8), (3, 50, 5), (40, 256, 32), (9, 2048, 256), (70, 136, 24), (2, 4096, 264)])
@pytest.mark.parametrize("mode", ["fp32", "bf16"])
def test_token_input_residual_and_next_norm(T, H, sd, mode):
    dtype, g = DT[mode], torch.Generator().manual_seed(T)
    r = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).float()
    V, L, i = 30, 3, 1
    x, delta, toks = torch.randn(T, H, generator=g), torch.randn(T, H, generator=g), torch.randint(0, V, (T,), generator=g)
    W = {"side.embed": r(V, L * sd), "side.gate": r(sd, H) / H ** 0.5, "side.proj": r(H, sd), "side.norm": r(H), "nw": r(H), "nb": r(H), "na": torch.tensor([0.75])}
    x1 = x + delta
    want_x = x1 + O.token_side(W, "", sd, i, 1e-5, x1, toks)
    want_h = O.dynamic_tanh(want_x, W["nw"], W["nb"], W["na"])
    P = {k: dev(v, dtype) for k, v in W.items()}
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    h = torch.empty(T, H, dtype=dtype, device="cuda")
    args = lambda xx, dd: (xx, dd, dev(toks, torch.int32), P["side.gate"], P["side.proj"], P["side.norm"], P["side.embed"], i, P["nw"], P["nb"], P["na"], h, 1e-5, status)
    C, tol = ext(), (2e-5 if mode == "fp32" else 0.01)
    gx = dev(x)
    C.side_fused(*args(gx, dev(delta)))
    close(gx, want_x, tol)
    close(h, want_h, tol)
    gx = dev(x1)
    z = (gx @ P["side.gate"].float().t()).contiguous()
    gg = torch.empty(T, sd, dtype=dtype, device="cuda")
    C.side_gate(*args(gx, None), z, gg)
    C.side_finish(*args(gx, None), (gg.float() @ P["side.proj"].float().t()).contiguous())
    close(gx, want_x, tol)
    close(h, want_h, tol)
    assert int(status) == 0


# ------------------------------------------------------------------------------------------------ latent attention
def latent_case(m, lens, news, seed, dtype, page=8, peak=4.0):
    """Cache rows of several sequences on shuffled pages, queries of their last ``news`` tokens, and what they should see."""
    g = torch.Generator().manual_seed(seed)
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    width = (R + r + 7) // 8 * 8
    q = lambda t: t.to(torch.bfloat16).float()
    ukv = q(torch.randn(H * (d + dv), R, generator=g) / R ** 0.5)
    pages_per = [(n + page - 1) // page for n in lens]
    perm = (torch.randperm(sum(pages_per), generator=g) + 1).tolist()
    rows = torch.full(((sum(pages_per) + 1) * page, width), float("nan"))
    table = torch.zeros(len(lens), max(pages_per) + 1, dtype=torch.int32)
    wants, qs, pos, seqs = [], [], [], []
    for b, (n, k) in enumerate(zip(lens, news)):
        own = [perm.pop() for _ in range(pages_per[b])]
        table[b, :len(own)] = torch.tensor(own, dtype=torch.int32)
        c, kr = q(torch.randn(n, R, generator=g)), q(torch.randn(n, r, generator=g))
        at = torch.arange(n)
        rows[torch.tensor(own)[at // page] * page + at % page] = torch.cat([c, kr, torch.zeros(n, width - R - r)], 1)
        qq = q(torch.randn(k, H, d + r, generator=g) * peak)   # sharp: single keys stand out
        for off, h in ((m["mask"]["size"], 0), (m["mask"]["size"] - 1, H - 1)):  # just outside and just inside the last query's window:
            if 0 <= n - 1 - off < n and (H > 1 or off == m["mask"]["size"]):                                             # keys that would take all of one head's weight
                v = ukv[h * d:(h + 1) * d].T @ qq[-1, h, :d]
                c[n - 1 - off] = q(3 * v / v.norm() * R ** 0.5)
        own_rows = torch.tensor(own)[at // page] * page + at % page
        rows[own_rows, :R] = c
        p = torch.arange(n - k, n)
        key = (c @ ukv[:H * d].T).view(n, H, d)
        val = (c @ ukv[H * d:].T).view(n, H, dv)
        s = (torch.einsum("ihd,jhd->hij", qq[..., :d], key) + torch.einsum("ihd,jd->hij", O.rotate(qq[..., d:], p, m["rot"]["base"]), kr)) * m["scale"]

        def attend(window):
            dist = p[:, None] - torch.arange(n)[None]
            a = torch.softmax(s.masked_fill(~((dist >= 0) & (dist < window)), float("-inf")), -1)
            return torch.einsum("hij,jhd->ihd", a, val).reshape(k, -1)

        wants.append((attend(m["mask"]["size"]), attend(m["mask"]["size"] + 1)))
        qs.append(qq.view(k, -1))
        pos += p.tolist()
        seqs += [b] * k
    rows = torch.where(torch.isnan(rows), torch.tensor(3.0e4), rows)  # (other slots: large, so that reading one shows)
    return dict(ukv=dev(ukv, dtype), rows=dev(rows, dtype), table=dev(table), q=dev(torch.cat(qs), dtype), pos=i32(pos), seqs=i32(seqs), page=page,
                want=torch.cat([w for w, _ in wants]), wrong=torch.cat([w for _, w in wants]), H=H, d=d, r=r, dv=dv)


def latent_args(m, c, status):
    from miles_b200.ops.reference import pair_frequencies

    freq = pair_frequencies(m["rot_dim"], m["rot"]["base"], "cuda")
    return (c["H"], c["d"], c["r"], c["dv"], m["mask"]["size"], m["scale"], c["ukv"], freq, c["rows"], c["table"], c["page"], status)


MIX = [dict(heads=4, dim=64, rot=32, vdim=64, kv_rank=64, window=130), dict(heads=20, dim=32, rot=16, vdim=48, kv_rank=128, window=64),
       dict(heads=3, dim=128, rot=64, vdim=128, kv_rank=512, window=200), dict(heads=1, dim=72, rot=8, vdim=80, kv_rank=72, window=1),
       dict(heads=33, dim=16, rot=8, vdim=8, kv_rank=40, window=129)]
ODD = [dict(heads=2, dim=9, rot=6, vdim=7, kv_rank=21, window=50), dict(heads=5, dim=12, rot=4, vdim=20, kv_rank=600, window=33)]


@pytest.mark.parametrize("spec", range(len(MIX) + len(ODD)))
@pytest.mark.parametrize("mode", ["fp32", "bf16"])
def test_decode_attention_over_pages_and_window_edges(spec, mode):
    C, m = ext(), latent(**(MIX + ODD)[spec])["mixer"]
    W = m["mask"]["size"]
    lens = [1, 2, 8, 9, W, W + 1, W + 2, max(1, W - 1), 2 * W + 5, 300]
    c = latent_case(m, lens, [1] * len(lens), spec, DT[mode])
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    tol = 3e-5 if mode == "fp32" else 0.03
    cat = torch.empty(len(lens), c["H"] * c["dv"] + 3, dtype=DT[mode], device="cuda")
    C.latent_attend(*latent_args(m, c, status), c["q"], c["pos"], None, cat)
    close(cat[:, :-3], c["want"], tol)
    assert (cat[:, :-3].float().cpu() - c["wrong"]).abs().max() > 0.3 * c["want"].abs().max()
    width = c["rows"].shape[1]
    if mode == "bf16" and C.latent_decode_supported(m["heads"], m["kv_rank"], m["rot_dim"], width):
        for splits in (1, 2, 5, 32):
            cat.fill_(float("nan"))
            C.latent_decode(*latent_args(m, c, status), c["q"], c["pos"], i32(lens), splits, cat)
            close(cat[:, :-3], c["want"], tol, splits)
    else:
        assert mode == "fp32" or spec >= len(MIX)
    assert int(status) == 0


@pytest.mark.parametrize("spec", range(len(MIX) + len(ODD)))
@pytest.mark.parametrize("mode", ["fp32", "bf16"])
def test_prompt_attention_in_portions_and_window_edges(spec, mode):
    C, m = ext(), latent(**(MIX + ODD)[spec])["mixer"]
    W = m["mask"]["size"]
    lens, news = [300, 5, W + 40, 131, 260, 2 * W + 3], [300, 5, 40, 2, 129, W + 3]
    c = latent_case(m, lens, news, 20 + spec, DT[mode])
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    tol = 3e-5 if mode == "fp32" else 0.03
    T = sum(news)
    ldc = (c["H"] * c["dv"] + 31) // 32 * 32
    cat = torch.empty(T, ldc, dtype=DT[mode], device="cuda")
    C.latent_attend(*latent_args(m, c, status), c["q"], c["pos"], c["seqs"], cat)
    close(cat[:, :c["H"] * c["dv"]], c["want"], tol)
    assert (cat[:, :c["H"] * c["dv"]].float().cpu() - c["wrong"]).abs().max() > 0.3 * c["want"].abs().max()
    if mode == "bf16" and C.latent_prefill_supported(m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], c["rows"].shape[1]):
        ranges, tiles, at, row = [], [], 0, 0
        for b, (n, k) in enumerate(zip(lens, news)):
            lo = max(0, n - k - W + 1)
            ranges.append((b, lo, at, n - lo))
            tiles += [(row + r, min(128, k - r), at, n - k - lo + r) for r in range(0, k, 128)]
            at, row = at + n - lo, row + k
        args = latent_args(m, c, status)
        lat = C.gather_rows(*args, i32(ranges), at, max(r[3] for r in ranges))
        kv = (lat[:, :m["kv_rank"]].float() @ c["ukv"].float().t()).to(torch.bfloat16).contiguous()
        cat.fill_(float("nan"))
        C.latent_prefill(*args, c["q"], c["pos"], lat, kv, i32(tiles), cat)
        close(cat[:, :c["H"] * c["dv"]], c["want"], 0.04)
    else:
        assert mode == "fp32" or spec >= len(MIX)
    assert int(status) == 0


def test_page_outside_the_cache_is_reported_not_followed():
    m = latent(**MIX[0])["mixer"]
    c = latent_case(m, [40], [1], 1, torch.bfloat16)
    c["table"][0, 2] = 10 ** 6
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    cat = torch.empty(1, c["H"] * c["dv"], dtype=torch.bfloat16, device="cuda")
    ext().latent_decode(*latent_args(m, c, status), c["q"], c["pos"], i32([40]), 1, cat)
    assert int(status) == 9 and torch.isfinite(cat.float()).all()


# ------------------------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module", params=[(k, m) for k in CASES for m in DT], ids=lambda p: "-".join(p))
def served(request, tmp_path_factory):
    name, mode = request.param
    cfg = CASES[name]
    W = O.random_weights(cfg, seed=3, dtype=torch.float32)
    eng = load(cfg, W, tmp_path_factory.mktemp("m"), "cuda", DT[mode], num_pages=200, max_seq_len=512)
    yield cfg, W, eng, DT[mode]
    eng.model.check_status()


def test_whole_prompt_single_tokens_and_portions(served):
    cfg, W, eng, dtype = served
    toks = tokens_of(301, cfg["vocab"], 1)
    want = O.model(cfg, W, toks)
    for cuts in ([301], [128, 2, 3, 100, 1], [7], [290, 1]):
        assert near(feed_all(eng, "a", toks, cuts), want, dtype), cuts
    assert near(feed_all(eng, "a", toks[:40], [2, 1]), want[:40], dtype)


def test_layers_one_by_one(served):
    cfg, W, eng, dtype = served
    toks, ref = tokens_of(40, cfg["vocab"], 5), []
    O.model(cfg, W, toks, ref)
    eng.model.capture = got = []
    t = i32(toks)
    eng.model.forward_hidden(t, torch.arange(40, dtype=torch.int32, device="cuda"), i32([0, 40]))
    eng.model.capture = None
    for i, (a, b) in enumerate(zip(got, ref)):
        close(a, b, 5e-5 if dtype == torch.float32 else 0.05, i)


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
        assert near(torch.cat([a for a, _ in rows]), torch.cat([b for _, b in rows]), dtype)
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
        ids = o["output_ids"]
        assert len(ids) == 60
        lg = O.model(cfg, W, p + ids[:-1])[len(p) - 1:]
        short = lg.max(-1).values - lg.gather(1, torch.tensor(ids)[:, None])[:, 0]
        assert short.max() < (1e-3 if dtype == torch.float32 else 0.3) * lg.std(), float(short.max() / lg.std())
    assert eng.pool.num_free == 33 and len(eng.slots_free) == 3


def test_plain_and_tensor_core_kernels_agree(tmp_path):
    cfg = CASES["tiles"]
    W = O.random_weights(cfg, seed=4, dtype=torch.float32)
    eng = load(cfg, W, tmp_path, "cuda", torch.bfloat16, num_pages=200, max_seq_len=512)
    toks = tokens_of(280, cfg["vocab"], 2)
    fast = feed_all(eng, "a", toks, [260, 1])
    eng.model.plain, eng.use_cuda_graph = True, False
    assert near(feed_all(eng, "b", toks, [260, 1]), fast, torch.bfloat16)


@pytest.mark.parametrize("mode", list(DT))
@pytest.mark.parametrize("window", [1, 63, 64, 65, 128, 129])
def test_window_edges_through_the_engine(tmp_path, mode, window):
    """Sharp attention: an oracle whose window is one longer is far away, in prompts, portions and decoding."""
    cfg = config([latent(heads=4, dim=32, rot=16, vdim=32, kv_rank=64, q_rank=64, window=window)])
    W = sharpen(cfg, O.random_weights(cfg, seed=window, dtype=torch.float32), 4.0)
    eng = load(cfg, W, tmp_path, "cuda", DT[mode], num_pages=100, max_seq_len=400, page_size=16)
    toks = tokens_of(300, cfg["vocab"], 4)
    want, wrong = O.model(cfg, W, toks), O.model(with_window(cfg, 1), W, toks)
    for cuts in ([300], [window + 1, 2], [250, 1]):
        got = feed_all(eng, "a", toks, cuts)
        assert row_errors(got, want).mean() < (5e-5 if mode == "fp32" else 0.02), cuts
        assert tells_apart(got, want, wrong)


def test_long_decoding_keeps_the_state_exact(tmp_path):
    cfg = config([mamba(heads=4, vdim=32, state=64), latent(window=50), mamba(heads=2, vdim=16, state=16, groups=1)])
    W = O.random_weights(cfg, seed=8, dtype=torch.float32)
    W["l0.mix.A_log"] = torch.full((4,), -7.0)
    for mode in DT:
        eng = load(cfg, W, tmp_path / mode, "cuda", DT[mode], num_pages=200, max_seq_len=900)
        toks = tokens_of(800, cfg["vocab"], 1)
        assert near(feed_all(eng, "a", toks, [2, 1]), O.model(cfg, W, toks), DT[mode])


def test_wide_decode_batch_takes_the_tensor_core_products(tmp_path):
    """More rows than the few-row kernels serve: products and token input run in their prompt form inside a decode step."""
    cfg = CASES["tiles"]
    W = O.random_weights(cfg, seed=4, dtype=torch.float32)
    eng = load(cfg, W, tmp_path, "cuda", torch.bfloat16, num_pages=1500, max_seq_len=64, max_running=300, page_size=8)
    seqs = {str(k): tokens_of(9 + k % 7, cfg["vocab"], k) for k in range(290)}
    eng.feed([(k, t[:-1], []) for k, t in seqs.items()])
    got = eng.feed([(k, t[-1:], [0]) for k, t in seqs.items()])
    pick = (0, 1, 137, 288, 289)
    assert near(torch.cat([got[k] for k in pick]).cpu(), torch.cat([O.model(cfg, W, seqs[str(k)])[-1:] for k in pick]), torch.bfloat16)
