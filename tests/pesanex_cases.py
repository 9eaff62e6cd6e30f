"""Small Pesanex configurations shared by the CPU and GPU tests (runners and error measures: rokivik_cases)."""
from __future__ import annotations

import copy

import torch


def retention(heads=2, dim=24, vdim=40, decay=None, dims=16, base=3000.0, ff=48):
    decay = decay or [1.0 - 2.0 ** -(1 + 2 * k % 9) for k in range(heads)]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": dims}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def gla(heads=3, dim=16, vdim=24, tau=8.0, ff=0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def parallel(heads=4, kv_heads=2, dim=16, vdim=24, dims=8, base=1000.0, scale=0.4, rheads=2, rdim=24, rvdim=16, tau=4.0, ff=56):
    return {"type": "parallel", "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                                   "rot": {"base": base, "dims": dims}},
                                          "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "tau": tau}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=64, vocab=96, eps=1e-5, loop=(0, 0, 1)):
    return {"architecture": "Pesanex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
            "loop": dict(zip(("start", "stop", "times"), loop))}


# rank of the projected decay, which the configuration does not say: by layer index
RANKS = {"odd": lambda i: 3 + 2 * i, "tiles": lambda i: 32 if i == 2 else 16}

CASES = {
    # every mixer, layers with and without a feed-forward, the loop in the middle
    "mixed": config([parallel(), retention(), gla(ff=40), parallel(heads=6, kv_heads=1, dims=16, ff=0)], loop=(1, 3, 2)),
    # sizes that no vector width or tile divides; the loop at the end, three times; rotation of 2 dimensions and of all of them
    "odd": config([gla(heads=1, dim=7, vdim=9, tau=3.0, ff=31), parallel(heads=3, kv_heads=3, dim=10, vdim=7, dims=10, rheads=5, rdim=3, rvdim=11, tau=1.0, ff=29),
                   retention(heads=3, dim=9, vdim=5, dims=2, ff=0)], width=50, vocab=61, eps=1e-3, loop=(1, 3, 3)),
    # widths the tensor maps take but no vector store does; the loop from the first layer
    "ragged": config([retention(heads=5, dim=8, vdim=24, dims=8, ff=37), gla(heads=3, dim=40, vdim=8, tau=16.0), parallel(heads=9, kv_heads=3, dim=40, vdim=72, dims=32)],
                     width=72, vocab=101, loop=(0, 2, 2)),
    # one kind of mixer only, without a loop
    "retained": config([retention(heads=4, dim=16, vdim=16, decay=[1.0, 0.5, 0.0, 0.999]), retention(heads=1, dim=32, vdim=64, dims=32)]),
    "gated": config([gla(), gla(heads=2, dim=32, vdim=32, tau=1.0, ff=64)], loop=(0, 2, 1)),
    # sizes the tensor-core kernels take
    "tiles": config([parallel(heads=8, kv_heads=2, dim=64, vdim=64, dims=32, scale=0.125, rheads=2, rdim=64, rvdim=64, ff=160),
                     retention(heads=2, dim=64, vdim=128, dims=64, ff=96), gla(heads=2, dim=128, vdim=128, tau=16.0),
                     parallel(heads=20, kv_heads=1, dim=128, vdim=128, dims=64, scale=0.1, rheads=3, rdim=48, rvdim=80, tau=16.0, ff=0),
                     parallel(heads=6, kv_heads=3, dim=96, vdim=112, dims=96, rheads=1, rdim=16, rvdim=32)], width=128, vocab=160, loop=(1, 4, 2)),
}


def sharpen(cfg, W, factor):
    """Attention that picks single keys out: larger scores."""
    c = copy.deepcopy(cfg)
    for l in c["layers"]:
        if l["type"] == "parallel":
            l["mixer"]["left"]["scale"] *= factor
    return c, W


def slow(W, names=("a2.b",), value=7.0):
    """Token decays near 1: what the first tokens left in the state stays."""
    return {k: torch.full_like(v, value) if k.endswith(names) else v for k, v in W.items()}
