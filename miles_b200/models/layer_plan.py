"""Per-layer descriptions for models whose layers are not all alike.

A ``LayerPlan`` lists, layer by layer, which mixer a decoder layer has (latent attention, Mamba-2, linear attention with a
fixed or a gated decay, softmax attention over key / value heads, two mixers side by side), that mixer's sizes and constants, and
its feed-forward; together with the model-wide choices (norm, residual arrangement, repeated layers, per-layer token input) it
is what parameter specs, checkpoint names, the cache layout and both execution paths are derived from. A ``ModelConfig`` with
``plan = None`` is the uniform attention + MLP decoder described by its flat fields.

Designs read from their own ``config.json`` register a reader in ``DESIGNS`` (keyed by the file's ``architecture``):

* ``Rokivik``: parallel layers (``x + mixer(h) + ff(h)`` over one Dynamic-Tanh norm), mixers ``mamba2`` and
  ``latent_attention`` in any order, an optional dense SwiGLU feed-forward, a gated per-layer token embedding after each.
* ``Pesanex``: two sublayers one after the other (``x + norm(mixer(norm(x)))``, then the same around an optional dense ReLU-gated
  feed-forward) with layer norms, mixers ``retention``, ``gla`` and ``parallel`` (softmax attention with sinks beside gated linear
  attention) in any order, a range of layers that runs several times with the same weights and a cache of its own each time.

Fused weights (``Segment`` lists below): everything that reads the layer's normed input is one matrix (mixer input rows |
gate rows | up rows), and everything that writes the residual is one matrix (mixer output columns | down columns), so a
parallel layer is two large products. Sequential layers have the mixer's input rows and the feed-forward's gate | up rows as one
matrix each. Segments start at multiples of 16 rows / 32 columns, which keeps every sub-view
aligned for vector loads and for the few-row product kernels.
"""
from __future__ import annotations

import json
import struct
from dataclasses import asdict, dataclass, field
from pathlib import Path
from typing import Optional, Union


def pad_to(n: int, a: int) -> int:
    return (n + a - 1) // a * a


@dataclass
class Rotary:
    """Rotary embedding of the first ``dims`` dimensions: pair k turns by ``position * base^(-2 k / dims)``. ``interleaved`` pairs
    dimension 2k with 2k + 1 (what the latent-attention kernels rotate), otherwise k with k + dims / 2 (what the other mixers do)."""
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
class LinearAttention:
    """Attention without a softmax: per head a state ``S <- diag(a) S + k v^T`` and an output ``S^T q``, whose root mean square is
    taken out, times ``silu(g)``. The decay ``a`` is one constant per head (``decay``) or, with ``rank`` > 0, comes from the token:
    ``sigmoid(W2 W1 h + bias)^(1 / tau)`` per key channel. The state is ``[heads, vdim, dim]`` fp32 per sequence."""
    heads: int
    dim: int
    vdim: int
    decay: Optional[list] = None          # one per head
    rank: int = 0                         # of the token's decay (0: ``decay``)
    tau: float = 1.0
    rotary: Optional[Rotary] = None       # of queries and keys
    scale_keys: bool = False              # dim^-1/2 belongs to the keys (after rotation), else to the queries
    norm_weight: bool = False             # the output norm has a weight [vdim], shared by the heads
    kind: str = "gla"

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.heads * self.dim

    @property
    def out_dim(self) -> int:
        return self.inner

    def in_parts(self) -> list:
        parts = [("v", self.inner), ("k", self.channels), ("q", self.channels), ("g", self.inner)]
        return parts + ([("a1", self.rank)] if self.rank else [])

    def out_parts(self) -> list:
        return [("o", self.out_dim)]

    def params(self) -> list:
        """(name, checkpoint leaf, shape, init) of what is not part of the fused matrices."""
        out = [("norm.weight", "norm", (self.vdim,), "ones")] if self.norm_weight else []
        if self.rank:
            out += [("a2.weight", "a2", (self.channels, self.rank), "normal"), ("a2.bias", "a2.b", (self.channels,), "zeros")]
        return out

    def check(self) -> None:
        if (self.decay is None) != bool(self.rank) or (self.decay is not None and len(self.decay) != self.heads):
            raise ValueError("linear attention needs one constant decay per head, or a projected one")
        if self.decay is not None and not all(0.0 <= d <= 1.0 for d in self.decay):
            raise ValueError("a decay lies between 0 and 1")
        if self.rank and not self.tau > 0:
            raise ValueError("tau must be positive")
        _check_halves(self.rotary, self.dim)


@dataclass
class Attention:
    """Causal softmax attention of ``heads`` query heads over ``kv_heads`` cached key / value heads. ``unit_qk``: rotated
    queries and keys are scaled to a root mean square of one. ``sink``: the softmax denominator has one more learned term per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rotary: Optional[Rotary] = None
    unit_qk: bool = False
    sink: bool = False
    kind: str = "attention"

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim

    @property
    def row_width(self) -> int:
        """Elements of one cached row: key heads, value heads, padding to 16 bytes of bf16."""
        return pad_to(self.kv_heads * (self.dim + self.vdim), 8)

    def in_parts(self) -> list:
        return [("q", self.heads * self.dim), ("k", self.kv_heads * self.dim), ("v", self.kv_heads * self.vdim)]

    def out_parts(self) -> list:
        return [("o", self.out_dim)]

    def params(self) -> list:
        return [("sink", "sink", (self.heads,), "zeros")] if self.sink else []

    def check(self) -> None:
        if self.kv_heads < 1 or self.heads % self.kv_heads:
            raise ValueError("key / value heads must divide the query heads")
        _check_halves(self.rotary, self.dim)


@dataclass
class Parallel:
    """Two mixers on the same input. Their outputs are RMS-normed, with a weight each, and averaged."""
    left: Union[Attention, LinearAttention]
    right: Union[Attention, LinearAttention]
    kind: str = "parallel"

    def sides(self) -> list:
        return [("left.", self.left), ("right.", self.right)]

    def in_parts(self) -> list:
        return [(p + n, s) for p, m in self.sides() for n, s in m.in_parts()]

    def out_parts(self) -> list:
        return [(p + n, s) for p, m in self.sides() for n, s in m.out_parts()]

    def params(self) -> list:
        return [(p + a, p + b, s, i) for p, m in self.sides() for a, b, s, i in m.params()]

    def check(self) -> None:
        self.left.check()
        self.right.check()


def _check_halves(r: Optional[Rotary], dim: int) -> None:
    if r is not None and (r.interleaved or r.dims % 2 or not 0 <= r.dims <= dim):
        raise NotImplementedError("heads are rotated in halves of an even number of leading dimensions")


@dataclass
class DenseFF:
    """Gated feed-forward: ``down(act(gate h) * (up h))``, act = silu or relu."""
    ff: int
    act: str = "silu"
    kind: str = "dense"


@dataclass
class Segment:
    name: str      # checkpoint leaf name
    start: int
    size: int


@dataclass
class Layer:
    mixer: Union[LatentAttention, Mamba2, LinearAttention, Attention, Parallel]
    ff: Optional[DenseFF] = None
    parallel: bool = True  # mixer and feed-forward read the same normed input (set by the plan)

    def in_segments(self) -> list:
        """Row ranges of the fused input matrix."""
        parts = [("mix." + n, s) for n, s in self.mixer.in_parts()]
        if self.ff is not None and self.parallel:
            parts += [("mlp.gate", self.ff.ff), ("mlp.up", self.ff.ff)]
        return _place(parts, 16)

    def out_segments(self) -> list:
        """Column ranges of the fused output matrix of a parallel layer."""
        parts = [("mix.o", self.mixer.out_dim)]
        if self.ff is not None:
            parts.append(("mlp.down", self.ff.ff))
        return _place(parts, 32)

    def ff_segments(self) -> list:
        """Row ranges of a sequential layer's feed-forward input matrix."""
        return _place([("mlp.gate", self.ff.ff), ("mlp.up", self.ff.ff)], 16)

    def out_matrices(self) -> list:
        """(parameter, checkpoint leaf, columns) of a sequential layer's mixer output matrices; their columns are padded to 32."""
        return [(n + ".weight", "mix." + n, size) for n, size in self.mixer.out_parts()]

    @property
    def in_rows(self) -> int:
        return seg_end(self.in_segments(), 16)

    @property
    def out_cols(self) -> int:
        return seg_end(self.out_segments(), 32)


def seg_end(segments: list, align: int) -> int:
    return pad_to(segments[-1].start + segments[-1].size, align)


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
    norm: str = "dynamic_tanh"       # the block norm and the final norm: dynamic_tanh, layer_norm (weight, no bias)
    eps: float = 1e-6
    # True: both sublayers read the same normed input and are added together. False: one after the other, each between a norm of
    # its input and a norm of its output
    parallel: bool = True
    token_side: int = 0              # width of the per-layer token input (0 = none)
    loop: Optional[tuple] = None     # (start, stop, times): layers start .. stop - 1 run that many times in a row

    def __post_init__(self):
        for l in self.layers:
            l.parallel = self.parallel

    def runs(self) -> list:
        """Layer indices in the order they run; every run has a cache of its own."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        start, stop, times = self.loop
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))

    def kv_source(self, i: int) -> int:
        """The layer whose latents layer ``i`` reads."""
        j = getattr(self.layers[i].mixer, "kv_from", None)
        return i if j is None else j

    def validate(self) -> None:
        assert self.layers, "a model needs at least one layer"
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start <= stop <= len(self.layers) or times < 1:
                raise ValueError(f"loop {self.loop} names no range of the {len(self.layers)} layers")
        if (self.norm, self.parallel, bool(self.token_side)) == ("layer_norm", False, False):
            for i, l in enumerate(self.layers):
                if not isinstance(l.mixer, (LinearAttention, Parallel)):
                    raise NotImplementedError(f"layer {i}: a {l.mixer.kind} mixer in a sequential block is not built")
                l.mixer.check()
                if isinstance(l.mixer, Parallel) and not (isinstance(l.mixer.left, Attention) and isinstance(l.mixer.right, LinearAttention)):
                    raise NotImplementedError(f"layer {i}: side by side run softmax attention and linear attention")
            return
        if self.norm != "dynamic_tanh" or not self.parallel or not self.token_side or self.loop is not None:
            raise NotImplementedError("planned layers are built as parallel blocks with Dynamic-Tanh norms and a per-layer token input, or as "
                                      "sequential blocks with layer norms")
        for i, l in enumerate(self.layers):
            m = l.mixer
            if l.ff is not None and l.ff.act != "silu":
                raise NotImplementedError(f"layer {i}: the feed-forward of a parallel block is gated by silu")
            if isinstance(m, Mamba2):
                if m.heads % m.groups or m.inner % m.norm_groups or m.conv < 1:
                    raise ValueError(f"layer {i}: groups must divide the heads and norm groups the inner width")
                continue
            if not isinstance(m, LatentAttention):
                raise NotImplementedError(f"layer {i}: a {m.kind} mixer in a parallel block is not built")
            if m.rotary.dims != m.rot_dim or m.rot_dim % 2 or not m.rotary.interleaved:
                raise NotImplementedError(f"layer {i}: latent attention rotates all {m.rot_dim} rotated dimensions, in interleaved pairs")
            if m.kv_from is not None:
                src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                if not isinstance(src, LatentAttention) or src.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from must name an earlier latent-attention layer with latents of its own")
                if (src.kv_rank, src.rot_dim, src.rotary) != (m.kv_rank, m.rot_dim, m.rotary):
                    raise ValueError(f"layer {i}: latents of layer {m.kv_from} have another size or rotation")


# ---------------------------------------------------------------------------------------------- readers / writers
def _read_rokivik(c: dict, shapes: dict) -> tuple:
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


# rank of the projected decay where neither the checkpoint's shapes nor the configuration say another
_DECAY_RANK = 16


def _read_pesanex(c: dict, shapes: dict) -> tuple:
    def rotary(m):
        return Rotary(base=float(m["rot"]["base"]), dims=int(m["rot"]["dims"]), interleaved=False)

    def sizes(m):
        return dict(heads=m["heads"], dim=m["dim"], vdim=m["vdim"])

    def gla(m, prefix):
        a1 = shapes.get(prefix + "a1")
        return LinearAttention(**sizes(m), rank=int(a1[0] if a1 is not None else m.get("rank", _DECAY_RANK)), tau=float(m["tau"]), norm_weight=True)

    layers = []
    for i, l in enumerate(c["layers"]):
        m, kind, p = l["mixer"], l["type"], f"l{i}.mix."
        if kind == "retention":
            mixer = LinearAttention(**sizes(m), decay=[float(d) for d in m["decay"]], rotary=rotary(m), scale_keys=True, kind=kind)
        elif kind == "gla":
            mixer = gla(m, p)
        elif kind == "parallel":
            a = m["left"]
            mixer = Parallel(Attention(**sizes(a), kv_heads=a["kv_heads"], scale=float(a["scale"]), rotary=rotary(a), unit_qk=True, sink=True),
                             gla(m["right"], p + "right."))
        else:
            raise NotImplementedError(f"mixer {kind!r} is not built")
        ff = l.get("mlp")
        if ff is not None and ff.get("kind") != "dense":
            raise NotImplementedError(f"feed-forward {ff.get('kind')!r} is not built")
        layers.append(Layer(mixer, DenseFF(ff["ff"], act="relu") if ff is not None else None))
    loop = c.get("loop")
    plan = LayerPlan("Pesanex", layers, norm="layer_norm", eps=float(c["norm"]["eps"]), parallel=False,
                     loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None)
    return plan, c["vocab"], c["width"]


def _write_pesanex(plan: LayerPlan, vocab: int, width: int) -> dict:
    def mixer(m):
        if isinstance(m, Parallel):
            return {"left": mixer(m.left), "right": mixer(m.right)}
        out = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim}
        if m.rotary is not None:
            out["rot"] = {"base": m.rotary.base, "dims": m.rotary.dims}
        if isinstance(m, Attention):
            out.update(kv_heads=m.kv_heads, scale=m.scale)
        elif m.decay is not None:
            out["decay"] = list(m.decay)
        else:
            out["tau"] = m.tau
            if m.rank != _DECAY_RANK:
                out["rank"] = m.rank
        return out

    c = {"architecture": plan.design, "norm": {"eps": plan.eps}, "vocab": vocab, "width": width,
         "layers": [{"type": l.mixer.kind, "mixer": mixer(l.mixer), "mlp": {"kind": "dense", "ff": l.ff.ff} if l.ff is not None else None} for l in plan.layers]}
    if plan.loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), plan.loop))
    return c


DESIGNS = {"Rokivik": (_read_rokivik, _write_rokivik), "Pesanex": (_read_pesanex, _write_pesanex)}


def checkpoint_shapes(path) -> dict:
    """name -> shape of every tensor in a directory's safetensors files, from their headers."""
    out = {}
    for f in sorted(Path(path).glob("*.safetensors")):
        with open(f, "rb") as fh:
            head = json.loads(fh.read(struct.unpack("<Q", fh.read(8))[0]))
        out.update({k: tuple(v["shape"]) for k, v in head.items() if k != "__metadata__"})
    return out


def read_plan(c: dict, shapes: Optional[dict] = None) -> tuple:
    """``config.json`` of a planned design -> (LayerPlan, vocabulary, width). ``shapes`` (name -> shape) of the checkpoint beside
    it give the sizes the configuration leaves to the tensors."""
    plan, vocab, width = DESIGNS[c["architecture"]][0](c, shapes or {})
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
        out.append((name + ".weight", (H,), "ones"))
        if plan.norm == "dynamic_tanh":
            out.extend([(name + ".bias", (H,), "zeros"), (name + ".alpha", (), "ones")])

    if first:
        out.append(("embed.weight", (vocab, H), "normal"))
    if sd:
        out.append(("side.embed.weight", (vocab, sd * len(plan.layers)), "normal"))
    for i in range(lo, hi):
        p, l = f"layers.{i}.", plan.layers[i]
        m = l.mixer
        norm(p + "norm1")
        out.append((p + "in.weight", (l.in_rows, H), "normal"))
        if not plan.parallel:
            out.extend((p + "mix." + n, shape, init) for n, _, shape, init in m.params())
            out.extend((p + n, (H, pad_to(size, 32)), "normal") for n, _, size in l.out_matrices())
            if isinstance(m, Parallel):
                norm(p + "mix.left.out_norm")
                norm(p + "mix.right.out_norm")
            norm(p + "norm1b")
            if l.ff is not None:
                norm(p + "norm2")
                out.extend([(p + "ff_in.weight", (seg_end(l.ff_segments(), 16), H), "normal"), (p + "ff_out.weight", (H, pad_to(l.ff.ff, 32)), "normal")])
                norm(p + "norm2b")
            continue
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
          "mix.uq.weight": "mix.uq", "norm1b.weight": "norm1b", "norm2.weight": "norm2", "norm2b.weight": "norm2b",
          "mix.left.out_norm.weight": "mix.left.out", "mix.right.out_norm.weight": "mix.right.out", "side.gate.weight": "side.gate", "side.proj.weight": "side.proj", "side.norm.weight": "side.norm"}
_TOP = {"embed.weight": "embed", "side.embed.weight": "side.embed", "lm_head.weight": "head", "final_norm.weight": "final.norm",
        "final_norm.bias": "final.norm.b", "final_norm.alpha": "final.norm.alpha"}


def plan_to_checkpoint(plan: LayerPlan, name: str, t) -> list:
    """One native tensor -> list of (checkpoint name, view of it)."""
    if name in _TOP:
        return [(_TOP[name], t)]
    _, idx, rest = name.split(".", 2)
    l, p = plan.layers[int(idx)], f"l{idx}."
    if not plan.parallel:
        for n, leaf, _, _ in l.mixer.params():
            if rest == "mix." + n:
                return [(p + "mix." + leaf, t)]
        for n, leaf, size in l.out_matrices():
            if rest == n:
                return [(p + leaf, t[:, :size])]
        if rest == "ff_in.weight":
            return [(p + s.name, t[s.start:s.start + s.size]) for s in l.ff_segments()]
        if rest == "ff_out.weight":
            return [(p + "mlp.down", t[:, :l.ff.ff])]
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
