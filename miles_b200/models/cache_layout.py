"""What a model keeps per token and per sequence while it generates.

The engine allocates, pages and hands out cache memory from this description instead of assuming one key and one value
tensor per layer: a layer may keep paged rows (one per cached token), state (one block per running sequence), nothing of
its own because it reads another layer's rows, or any mix of these.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from .layer_plan import Attention, LinearAttention, Mamba2, Parallel


@dataclass
class LayerCache:
    paged: list = field(default_factory=list)      # (shape of one token's row, dtype)
    state: list = field(default_factory=list)      # (shape of one sequence's state, dtype)
    shares: Optional[int] = None                   # use this layer's tensors


@dataclass
class CacheLayout:
    layers: list

    @property
    def has_state(self) -> bool:
        return any(l.state for l in self.layers)

    @staticmethod
    def _bytes(items: list) -> int:
        n = 0
        for shape, dtype in items:
            k = torch.empty((), dtype=dtype).element_size()
            for s in shape:
                k *= s
            n += k
        return n

    def bytes_per_slot(self) -> int:
        return sum(self._bytes(l.paged) for l in self.layers)

    def bytes_per_sequence(self) -> int:
        return sum(self._bytes(l.state) for l in self.layers)

    def allocate(self, slots: int, sequences: int, device, storage: Optional[torch.Tensor] = None) -> list:
        """Per layer a tuple of tensors: paged ones ``[slots, ...]`` first, then state ``[sequences, ...]``. With
        ``storage`` (uint8, contents undefined) the paged tensors are carved out of it; state is always allocated."""
        out, at = [], 0
        for l in self.layers:
            if l.shares is not None:
                out.append(out[l.shares])
                continue
            ts = []
            for shape, dtype in l.paged:
                if storage is None:
                    ts.append(torch.zeros((slots,) + tuple(shape), dtype=dtype, device=device))
                    continue
                n = slots * self._bytes([(shape, dtype)])
                assert storage.numel() >= at + n, "the storage for the paged cache is too small"
                ts.append(storage[at:at + n].view(dtype).view((slots,) + tuple(shape)))
                at += n
            ts += [torch.zeros((sequences,) + tuple(shape), dtype=dtype, device=device) for shape, dtype in l.state]
            out.append(tuple(ts))
        return out


def _mixer_cache(m, dtype: torch.dtype) -> LayerCache:
    """What one mixer keeps: latent attention one row (latent | rotated key part) per token; softmax attention one row (keys |
    values) per token; Mamba-2 the last ``conv`` inputs of its convolution as a ring indexed by position (one more than it reads
    back, so that writing a token's input never touches what is read for it) and the fp32 state ``[heads, vdim, state]``; linear
    attention the fp32 state ``[heads, vdim, dim]``; two mixers side by side what each of them does."""
    if isinstance(m, Mamba2):
        return LayerCache(state=[((m.conv, m.channels), dtype), ((m.heads, m.vdim, m.state), torch.float32)])
    if isinstance(m, LinearAttention):
        return LayerCache(state=[((m.heads, m.vdim, m.dim), torch.float32)])
    if isinstance(m, Attention):
        return LayerCache(paged=[((m.row_width,), dtype)])
    if isinstance(m, Parallel):
        a, b = _mixer_cache(m.left, dtype), _mixer_cache(m.right, dtype)
        return LayerCache(paged=a.paged + b.paged, state=a.state + b.state)
    return LayerCache(paged=[((m.latent_width,), dtype)])


def cache_layout(cfg, dtype: torch.dtype) -> CacheLayout:
    """The cache of a model: keys and values per layer, or whatever the mixers of its layer plan keep, one entry per run of a
    layer (layers that run several times keep something for each pass)."""
    if cfg.plan is None:
        kv = [((cfg.num_kv_heads, cfg.head_dim), dtype)] * 2
        return CacheLayout([LayerCache(paged=kv) for _ in range(cfg.num_layers)])
    layers = []
    for i in cfg.plan.runs():
        m = cfg.plan.layers[i].mixer
        src = getattr(m, "kv_from", None)
        layers.append(LayerCache(shares=src) if src is not None else _mixer_cache(m, dtype))
    return CacheLayout(layers)
