"""Per-layer descriptions for models whose layers are not all alike.

A ``LayerPlan`` lists, layer by layer, which mixer a decoder layer has (latent attention, Mamba-2), that mixer's sizes and
constants, and its feed-forward; together with the model-wide choices (norm, residual arrangement, per-layer token input)
it is what parameter specs, checkpoint names, the cache layout and both execution paths are derived from. A ``ModelConfig``
with ``plan = None`` is the uniform attention + MLP decoder described by its flat fields.

Designs read from their own ``config.json`` register a reader in ``DESIGNS`` (keyed by the file's ``architecture``):

* ``Rokivik``: parallel layers (``x + mixer(h) + ff(h)`` over one Dynamic-Tanh norm), mixers ``mamba2`` and
  ``latent_attention`` in any order, an optional dense SwiGLU feed-forward, a gated per-layer token embedding after each.

Fused weights (``Segment`` lists below): everything that reads the layer's normed input is one matrix (mixer input rows |
gate rows | up rows), and everything that writes the residual is one matrix (mixer output columns | down columns), so a
parallel layer is two large products. Segments start at multiples of 16 rows / 32 columns, which keeps every sub-view
aligned for vector loads and for the few-row product kernels.
"""
from __future__ import annotations

from dataclasses import asdict, dataclass, field
from typing import Optional, Union


def pad_to(n: int, a: int) -> int:
    return (n + a - 1) // a * a


@dataclass
class Rotary:
    """Rotary embedding of ``dims`` dimensions: pair k turns by ``position * base^(-2 k / dims)``. ``interleaved`` pairs
    dimension 2k with 2k + 1 (the only arrangement the latent-attention kernels rotate)."""
    base: float = 10000.0
    dims: int = 64
    interleaved: bool = True


@dataclass
class LatentAttention:
    """Multi-head attention whose keys and values are projections of one small latent per token (plus one rotated key
    part shared by all heads); only latent and rotated part are cached. ``window`` > 0: a query sees itself and the
    ``window - 1`` tokens before it; 0: all earlier tokens. ``kv_from``: use that layer's cached latents instead of
    projecting own ones."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    window: int = 0
    rotary: Rotary = field(default_factory=Rotary)
    kv_from: Optional[int] = None
    kind: str = "latent_attention"

    @property
    def q_dim(self) -> int:
        return self.heads * (self.dim + self.rot_dim)

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def latent_width(self) -> int:
        """Elements of one cached row: latent, rotated key part, padding to 16 bytes of bf16."""
        return pad_to(self.kv_rank + self.rot_dim, 8)

    def in_parts(self) -> list:
        parts = [("dq", self.q_rank)]
        if self.kv_from is None:
            parts.append(("dkv", self.kv_rank + self.rot_dim))
        return parts


@dataclass
class Mamba2:
    """Mamba-2 mixer: gated selective state space with a short causal convolution in front. The state is
    ``[heads, vdim, state]`` per sequence plus the convolution's last inputs."""
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int
    kind: str = "mamba2"

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    @property
    def out_dim(self) -> int:
        return self.inner

    def in_parts(self) -> list:
        return [("in", self.inner + self.channels + self.heads)]


@dataclass
class DenseFF:
    """SwiGLU feed-forward: ``down(silu(gate h) * (up h))``."""
    ff: int
    kind: str = "dense"


@dataclass
class Segment:
    name: str      # checkpoint leaf name
    start: int
    size: int


@dataclass
class Layer:
    mixer: Union[LatentAttention, Mamba2]
    ff: Optional[DenseFF] = None

    def in_segments(self) -> list:
        """Row ranges of the fused input matrix."""
        parts = [("mix." + n, s) for n, s in self.mixer.in_parts()]
        if self.ff is not None:
            parts += [("mlp.gate", self.ff.ff), ("mlp.up", self.ff.ff)]
        return _place(parts, 16)

    def out_segments(self) -> list:
        """Column ranges of the fused output matrix."""
        parts = [("mix.o", self.mixer.out_dim)]
        if self.ff is not None:
            parts.append(("mlp.down", self.ff.ff))
        return _place(parts, 32)

    @property
    def in_rows(self) -> int:
        s = self.in_segments()[-1]
        return pad_to(s.start + s.size, 16)

    @property
    def out_cols(self) -> int:
        s = self.out_segments()[-1]
        return pad_to(s.start + s.size, 32)


def _place(parts: list, align: int) -> list:
    out, at = [], 0
    for name, size in parts:
        out.append(Segment(name, at, size))
        at = pad_to(at + size, align)
    return out


@dataclass
class LayerPlan:
    design: str
    layers: list
    norm: str = "dynamic_tanh"       # the block norm and the final norm
    eps: float = 1e-6
    parallel: bool = True            # both sublayers read the same normed input and are added together
    token_side: int = 0              # width of the per-layer token input (0 = none)

    def kv_source(self, i: int) -> int:
        """The layer whose latents layer ``i`` reads."""
        j = getattr(self.layers[i].mixer, "kv_from", None)
        return i if j is None else j

    @property
    def has_state(self) -> bool:
        return any(isinstance(l.mixer, Mamba2) for l in self.layers)

    def validate(self) -> None:
        assert self.layers, "a model needs at least one layer"
        if self.norm != "dynamic_tanh" or not self.parallel or not self.token_side:
            raise NotImplementedError("planned layers are built for parallel blocks with Dynamic-Tanh norms and a per-layer token input")
        for i, l in enumerate(self.layers):
            m = l.mixer
            if isinstance(m, Mamba2):
                if m.heads % m.groups or m.inner % m.norm_groups or m.conv < 1:
                    raise ValueError(f"layer {i}: groups must divide the heads and norm groups the inner width")
                continue
            if m.rotary.dims != m.rot_dim or m.rot_dim % 2 or not m.rotary.interleaved:
                raise NotImplementedError(f"layer {i}: latent attention rotates all {m.rot_dim} rotated dimensions, in interleaved pairs")
            if m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if not isinstance(src, LatentAttention) or src.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from must name an earlier latent-attention layer with latents of its own")
                if (src.kv_rank, src.rot_dim, src.rotary) != (m.kv_rank, m.rot_dim, m.rotary):
                    raise ValueError(f"layer {i}: latents of layer {m.kv_from} have another size or rotation")


# ---------------------------------------------------------------------------------------------- readers / writers
def _read_rokivik(c: dict) -> tuple:
    layers = []
    for l in c["layers"]:
        m, kind = l["mixer"], l["type"]
        if kind == "mamba2":
            mixer = Mamba2(heads=m["heads"], vdim=m["vdim"], state=m["state"], groups=m["groups"], conv=m["conv"], norm_groups=m["norm_groups"])
        elif kind == "latent_attention":
            rot = m["rot"]
            mixer = LatentAttention(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"],
                                    q_rank=m["q_rank"], scale=float(m["scale"]), window=int((m.get("mask") or {}).get("size", 0)),
                                    rotary=Rotary(base=float(rot["base"]), dims=int(rot["dims"])), kv_from=m.get("kv_from"))
        else:
            raise NotImplementedError(f"mixer {kind!r} is not built")
        ff = l.get("mlp")
        if ff is not None and ff.get("kind") != "dense":
            raise NotImplementedError(f"feed-forward {ff.get('kind')!r} is not built")
        layers.append(Layer(mixer, DenseFF(ff["ff"]) if ff is not None else None))
    plan = LayerPlan("Rokivik", layers, eps=float(c["norm"]["eps"]), token_side=int(c["token_side"]["dim"]))
    return plan, c["vocab"], c["width"]


def _write_rokivik(plan: LayerPlan, vocab: int, width: int) -> dict:
    layers = []
    for l in plan.layers:
        m = asdict(l.mixer)
        kind = m.pop("kind")
        if kind == "latent_attention":
            rot, window, src = m.pop("rotary"), m.pop("window"), m.pop("kv_from")
            m["rot"] = {"base": rot["base"], "dims": rot["dims"]}
            if window:
                m["mask"] = {"size": window}
            if src is not None:
                m["kv_from"] = src
        layers.append({"type": kind, "mixer": m, "mlp": {"kind": "dense", "ff": l.ff.ff} if l.ff is not None else None})
    return {"architecture": plan.design, "layers": layers, "norm": {"eps": plan.eps}, "token_side": {"dim": plan.token_side},
            "vocab": vocab, "width": width}


DESIGNS = {"Rokivik": (_read_rokivik, _write_rokivik)}


def read_plan(c: dict) -> tuple:
    """``config.json`` of a planned design -> (LayerPlan, vocabulary, width)."""
    plan, vocab, width = DESIGNS[c["architecture"]][0](c)
    plan.validate()
    return plan, int(vocab), int(width)


def write_plan(plan: LayerPlan, vocab: int, width: int) -> dict:
    return DESIGNS[plan.design][1](plan, vocab, width)


# ---------------------------------------------------------------------------------------------- parameters
def plan_specs(plan: LayerPlan, vocab: int, width: int, lo: int, hi: int, first: bool, last: bool) -> list:
    """(name, shape, init) of every parameter of layers ``lo..hi``."""
    H, sd = width, plan.token_side
    out = []

    def norm(name: str) -> None:
        out.extend([(name + ".weight", (H,), "ones"), (name + ".bias", (H,), "zeros"), (name + ".alpha", (), "ones")])

    if first:
        out.append(("embed.weight", (vocab, H), "normal"))
    out.append(("side.embed.weight", (vocab, sd * len(plan.layers)), "normal"))
    for i in range(lo, hi):
        p, l = f"layers.{i}.", plan.layers[i]
        m = l.mixer
        norm(p + "norm1")
        out.append((p + "in.weight", (l.in_rows, H), "normal"))
        if isinstance(m, Mamba2):
            out.extend([(p + "mix.conv.weight", (m.channels, m.conv), "normal"), (p + "mix.conv.bias", (m.channels,), "zeros"),
                        (p + "mix.dt_bias", (m.heads,), "zeros"), (p + "mix.A_log", (m.heads,), "zeros"), (p + "mix.D", (m.heads,), "ones"),
                        (p + "mix.norm.weight", (m.inner,), "ones")])
        else:
            out.append((p + "mix.q_norm.weight", (m.q_rank,), "ones"))
            if m.kv_from is None:
                out.append((p + "mix.kv_norm.weight", (m.kv_rank,), "ones"))
            out.extend([(p + "mix.uq.weight", (m.q_dim, m.q_rank), "normal"),
                        (p + "mix.ukv.weight", (m.heads * (m.dim + m.vdim), m.kv_rank), "normal")])
        out.append((p + "out.weight", (H, l.out_cols), "normal"))
        out.extend([(p + "side.gate.weight", (sd, H), "normal"), (p + "side.proj.weight", (H, sd), "normal"),
                    (p + "side.norm.weight", (H,), "ones")])
    if last:
        norm("final_norm")
        out.append(("lm_head.weight", (vocab, H), "normal"))
    return out


_PLAIN = {"norm1.weight": "norm1", "norm1.bias": "norm1.b", "norm1.alpha": "norm1.alpha", "mix.conv.weight": "mix.conv",
          "mix.conv.bias": "mix.conv.b", "mix.dt_bias": "mix.dt_bias", "mix.A_log": "mix.A_log", "mix.D": "mix.D",
          "mix.norm.weight": "mix.norm", "mix.q_norm.weight": "mix.dq.norm", "mix.kv_norm.weight": "mix.dkv.norm",
          "mix.uq.weight": "mix.uq", "side.gate.weight": "side.gate", "side.proj.weight": "side.proj", "side.norm.weight": "side.norm"}
_TOP = {"embed.weight": "embed", "side.embed.weight": "side.embed", "lm_head.weight": "head", "final_norm.weight": "final.norm",
        "final_norm.bias": "final.norm.b", "final_norm.alpha": "final.norm.alpha"}


def plan_to_checkpoint(plan: LayerPlan, name: str, t) -> list:
    """One native tensor -> list of (checkpoint name, view of it)."""
    if name in _TOP:
        return [(_TOP[name], t)]
    _, idx, rest = name.split(".", 2)
    l, p = plan.layers[int(idx)], f"l{idx}."
    if rest in _PLAIN:
        return [(p + _PLAIN[rest], t)]
    if rest == "in.weight":
        return [(p + s.name, t[s.start:s.start + s.size]) for s in l.in_segments()]
    if rest == "out.weight":
        return [(p + s.name, t[:, s.start:s.start + s.size]) for s in l.out_segments()]
    if rest == "mix.ukv.weight":
        k = l.mixer.heads * l.mixer.dim
        return [(p + "mix.uk", t[:k]), (p + "mix.uv", t[k:])]
    raise KeyError(name)
