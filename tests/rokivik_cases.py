"""Small Rokivik configurations and runners shared by the CPU and GPU tests."""
from __future__ import annotations

import torch

import oracle_rokivik as O


def mamba(heads=4, vdim=16, state=16, groups=2, conv=4, norm_groups=2, ff=48):
    return {"type": "mamba2", "mixer": dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups),
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads=3, dim=16, rot=8, vdim=24, kv_rank=32, q_rank=40, window=9, base=1000.0, scale=None, ff=48, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale or (dim + rot) ** -0.5,
             mask={"size": window}, rot={"base": base, "dims": rot})
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=64, vocab=96, side=8, eps=1e-5):
    return {"architecture": "Rokivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "token_side": {"dim": side}, "layers": layers}


CASES = {
    # mixed order, a layer reading another's latents with its own heads and window, a layer without a feed-forward
    "mixed": config([mamba(), latent(), mamba(ff=0), latent(heads=5, dim=24, vdim=16, window=70, kv_from=1, ff=0), latent(kv_rank=48, rot=16, window=33)]),
    # sizes that no vector width or tile divides, one group, one head, taps and windows of other lengths, side width 5
    "odd": config([latent(heads=1, dim=10, rot=6, vdim=7, kv_rank=19, q_rank=13, window=1, ff=31), mamba(heads=3, vdim=5, state=7, groups=1, conv=3, norm_groups=3, ff=29),
                   latent(heads=2, dim=9, rot=4, vdim=11, kv_rank=21, q_rank=17, window=13, ff=0), mamba(heads=6, vdim=9, state=33, groups=3, conv=6, norm_groups=1, ff=17)],
                  width=50, vocab=61, side=5, eps=1e-3),
    # widths the tensor maps take but no vector store does (odd row counts of weights, an odd vocabulary)
    "ragged": config([latent(heads=3, dim=24, rot=8, vdim=8, kv_rank=40, q_rank=24, window=21, ff=37), mamba(heads=5, vdim=8, state=8, groups=5, norm_groups=5, ff=23),
                      latent(heads=1, dim=40, rot=16, vdim=72, kv_rank=136, q_rank=8, window=300, ff=0)], width=72, vocab=101, side=16),
    # recurrence only / attention only
    "recurrent": config([mamba(heads=2, vdim=32, state=64, groups=1, norm_groups=1), mamba(conv=2)]),
    "attention": config([latent(window=17), latent(window=40, kv_from=0, scale=0.9)]),
    # sizes the tensor-core kernels take
    "tiles": config([mamba(heads=4, vdim=64, state=128, groups=2, norm_groups=4, ff=160),
                     latent(heads=4, dim=64, rot=32, vdim=64, kv_rank=64, q_rank=64, window=150, ff=160),
                     mamba(heads=8, vdim=32, state=64, groups=1, norm_groups=1, ff=160),
                     latent(heads=18, dim=96, rot=16, vdim=80, kv_rank=64, q_rank=96, window=64, ff=160, base=50000.0),
                     latent(heads=2, dim=128, rot=32, vdim=128, kv_rank=64, q_rank=64, window=260, ff=160, kv_from=1)], width=128, vocab=160, side=32),
}


def load(cfg, W, tmp_path, device, dtype, **engine_kw):
    """(engine, model) serving the checkpoint written from ``W`` through the framework's own configuration and loader."""
    from miles_b200.checkpoint import load_hf
    from miles_b200.engine import Engine
    from miles_b200.models import ParamStore, build_model, get_config

    d = O.write_checkpoint(tmp_path, cfg, W)
    mc = get_config(str(d))
    store = ParamStore(mc, device, dtype)  # (random first: every value must come from the checkpoint)
    assert load_hf(mc, store, str(d)) == len(W)
    kw = dict(max_running=4, num_pages=64, page_size=8, max_seq_len=256, max_prefill_tokens=4096)
    kw.update(engine_kw)
    return Engine(build_model(mc, store), **kw)


def tokens_of(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def feed_all(eng, rid, toks, cuts, end=True):
    """Logits [len(toks), vocab] of a sequence fed in portions of the given sizes (the last size repeats)."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        out.append(eng.feed([(rid, toks[at:at + n], list(range(n)))])[0].float().cpu())
        at, k = at + n, k + 1
    if end:
        eng.end_feed(rid)
    return torch.cat(out)


def row_errors(a, b):
    """Error of every row (mean over the vocabulary taken off, root mean square) over the spread of the logits."""
    a, b = a.double(), b.double()
    d = a - b
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / b.std()


def rel(a, b):
    return float(row_errors(a, b).max())


def near(a, b, dtype):
    """Logits agree up to rounding: every row in 32-bit; in bf16 (where a sharp softmax row can turn on one rounding) the
    mean of the rows closely and the worst row loosely."""
    e = row_errors(a, b)
    if dtype == torch.float32:
        return bool(e.max() < 5e-5)
    return bool(e.mean() < 0.02 and e.max() < 0.25)


def tells_apart(got, want, wrong):
    """Where the two references differ most, ``got`` follows ``want``."""
    r = int(row_errors(wrong, want).argmax())
    return float(row_errors(got[r:r + 1], want[r:r + 1])) < 0.3 * float(row_errors(got[r:r + 1], wrong[r:r + 1]))


def sharpen(cfg, W, factor):
    """Attention that picks single keys out: queries scaled up, so that one far key decides a row."""
    W = dict(W)
    for name in W:
        if name.endswith("mix.uq"):
            W[name] = (W[name] * factor).to(torch.bfloat16).to(W[name].dtype)
    return W


def with_window(cfg, delta):
    """The same configuration with every window longer by ``delta`` (for the oracle's planted mistake)."""
    import copy

    c = copy.deepcopy(cfg)
    for l in c["layers"]:
        if "mask" in l["mixer"]:
            l["mixer"]["mask"]["size"] += delta
    return c
