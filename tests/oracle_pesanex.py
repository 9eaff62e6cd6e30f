"""Plain restatement of the Pesanex equations, one function per mechanism, token by token where that is the clearest form.
Tests compare the product with it; it imports nothing from the package.

Weights are a dict ``name -> tensor`` under the checkpoint's names, ``cfg`` the parsed ``config.json``. Everything is
computed in the dtype of the tensors it is given (tests use float32 or float64)."""
from __future__ import annotations

import torch


# ------------------------------------------------------------------------------------------- small functions
def silu(z):
    return z / (1 + torch.exp(-z))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rotate_half(x, positions, base, dims):
    """``x`` [T, heads, dim]: dimensions i and i + dims / 2 are turned by position * base^(-2i / dims), i < dims / 2."""
    out, half = x.clone(), dims // 2
    for i in range(half):
        a = (positions.double() * base ** (-2.0 * i / dims)).view(-1, 1)
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------- recurrences
def recurrence(q, k, v, alpha):
    """``S <- diag(alpha_t) S + k_t v_t^T, o_t = S^T q_t`` per head: q, k, alpha [T, H, N], v [T, H, P]."""
    S = q.new_zeros(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, q[t]))
    return torch.stack(out)


def retention(W, p, m, eps, h, positions):
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate_half((h @ W[p + "q"].T).view(T, H, N), positions, m["rot"]["base"], m["rot"]["dims"])
    k = rotate_half((h @ W[p + "k"].T).view(T, H, N), positions, m["rot"]["base"], m["rot"]["dims"]) * N ** -0.5
    alpha = torch.tensor(m["decay"], dtype=torch.float64).to(h.dtype).view(1, H, 1).expand(T, H, N)
    o = unit_rms(recurrence(q, k, (h @ W[p + "v"].T).view(T, H, P), alpha), eps).reshape(T, H * P)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def channel_decay(W, p, m, h):
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    return torch.exp(torch.nn.functional.logsigmoid(z) / m["tau"]).view(h.shape[0], m["heads"], m["dim"])


def gated_linear(W, p, m, eps, h, positions=None):
    T, H, N, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ W[p + n].T).view(T, H, -1) for n in "qkv")
    o = unit_rms(recurrence(q * N ** -0.5, k, v, channel_decay(W, p, m, h)), eps) * W[p + "norm"]
    return (o.reshape(T, H * P) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------- attention
def sink_softmax(s, sink):
    """Weights over the last dimension of ``s`` [H, T, T'] with one more term exp(sink_h) in the denominator."""
    top = torch.maximum(s.max(-1, keepdim=True).values, sink.view(-1, 1, 1))
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink.view(-1, 1, 1) - top))


def attention(W, p, m, eps, h, positions):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    turn = lambda x: unit_rms(rotate_half(x, positions, m["rot"]["base"], m["rot"]["dims"]), eps)
    q = turn((h @ W[p + "q"].T).view(T, H, m["dim"]))
    k = turn((h @ W[p + "k"].T).view(T, G, m["dim"])).repeat_interleave(H // G, 1)
    v = (h @ W[p + "v"].T).view(T, G, m["vdim"]).repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], float("-inf"))
    return torch.einsum("hij,jhd->ihd", sink_softmax(s, W[p + "sink"]), v).reshape(T, -1) @ W[p + "o"].T


def side_by_side(W, p, m, eps, h, positions):
    a = unit_rms(attention(W, p + "left.", m["left"], eps, h, positions), eps) * W[p + "left.out"]
    b = unit_rms(gated_linear(W, p + "right.", m["right"], eps, h), eps) * W[p + "right.out"]
    return (a + b) / 2


MIXERS = {"retention": retention, "gla": gated_linear, "parallel": side_by_side}


def dense_ff(W, p, h):
    return (torch.clamp(h @ W[p + "gate"].T, min=0) * (h @ W[p + "up"].T)) @ W[p + "down"].T


# ------------------------------------------------------------------------------------------- the model
def layer_order(cfg):
    n, loop = len(cfg["layers"]), cfg["loop"]
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


def model(cfg, W, tokens, residuals=None):
    """Logits [T, vocab] of one sequence; ``residuals`` (a list) receives the residual stream after every layer run."""
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(tokens).long()
    positions = torch.arange(len(tokens))
    x = W["embed"][tokens]
    for i in layer_order(cfg):
        p, layer = f"l{i}.", cfg["layers"][i]
        y = MIXERS[layer["type"]](W, p + "mix.", layer["mixer"], eps, layer_norm(x, W[p + "norm1"], eps), positions)
        x = x + layer_norm(y, W[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            x = x + layer_norm(dense_ff(W, p + "mlp.", layer_norm(x, W[p + "norm2"], eps)), W[p + "norm2b"], eps)
        if residuals is not None:
            residuals.append(x)
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T


# ------------------------------------------------------------------------------------------- checkpoints for tests
def tensor_shapes(cfg, rank=None):
    """name -> shape of every tensor of a checkpoint with this configuration. The rank of the decay's projection is no key
    of the configuration: ``rank(layer index)``."""
    V, H = cfg["vocab"], cfg["width"]
    rank = rank or (lambda i: 16)
    out = {"embed": (V, H), "head": (V, H), "final.norm": (H,)}

    def linear(p, m, i, gated):
        n, v = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        out.update({p + "q": (n, H), p + "k": (n, H), p + "v": (v, H), p + "g": (v, H), p + "o": (H, v)})
        if gated:
            out.update({p + "norm": (m["vdim"],), p + "a1": (rank(i), H), p + "a2": (n, rank(i)), p + "a2.b": (n,)})

    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] is not None else ()):
            out[p + n] = (H,)
        if layer["type"] == "parallel":
            a, q = m["left"], p + "mix.left."
            out.update({q + "q": (a["heads"] * a["dim"], H), q + "k": (a["kv_heads"] * a["dim"], H), q + "v": (a["kv_heads"] * a["vdim"], H),
                        q + "sink": (a["heads"],), q + "o": (H, a["heads"] * a["vdim"]), q + "out": (H,)})
            linear(p + "mix.right.", m["right"], i, True)
            out[p + "mix.right.out"] = (H,)
        else:
            linear(p + "mix.", m, i, layer["type"] == "gla")
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            out.update({p + "mlp.gate": (f, H), p + "mlp.up": (f, H), p + "mlp.down": (H, f)})
    return out


def random_weights(cfg, seed=0, dtype=torch.bfloat16, rank=None):
    """Random bf16-representable weights with scales at which every branch matters."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf.startswith("norm") or leaf == "out":
            t = 1 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "b":
            t = 1 + 2 * torch.randn(shape, generator=g)
        elif leaf == "sink":
            t = torch.randn(shape, generator=g)
        elif leaf == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
        W[name] = t.to(torch.bfloat16).to(dtype)
    return W
