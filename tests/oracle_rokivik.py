"""Plain fp32 / fp64 restatement of the Rokivik equations, one function per mechanism, token by token where that is the
clearest form. Tests compare the product with it; it imports nothing from the package.

Weights are a dict ``name -> tensor`` under the checkpoint's names, ``cfg`` the parsed ``config.json``. Everything is
computed in the dtype of the tensors it is given (tests use float32 or float64)."""
from __future__ import annotations

import json
import math
import struct

import torch


# ------------------------------------------------------------------------------------------- small functions
def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def dynamic_tanh(x, w, b, alpha):
    return torch.tanh(alpha * x) * w + b


def rotate(x, positions, base):
    """``x`` [T, ..., R]: pairs (2i, 2i + 1) turned by position * base^(-2i / R)."""
    R = x.shape[-1]
    out = x.clone()
    for i in range(R // 2):
        a = (positions.to(x.dtype) * base ** (-2.0 * i / R)).view(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


# ------------------------------------------------------------------------------------------- latent attention
def latent_of(W, p, m, eps, h, positions):
    """What a latent-attention layer remembers of every token: the normed latent and the rotated shared key part."""
    t = h @ W[p + "dkv"].T
    c = unit_rms(t[:, :m["kv_rank"]], eps) * W[p + "dkv.norm"]
    return c, rotate(t[:, m["kv_rank"]:], positions, m["rot"]["base"])


def latent_attention(W, p, m, eps, h, positions, c, kr):
    T, H, d, r, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    cq = unit_rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (cq @ W[p + "uq"].T).view(T, H, d + r)
    qn, qr = q[..., :d], rotate(q[..., d:], positions, m["rot"]["base"])
    k = (c @ W[p + "uk"].T).view(T, H, d)
    v = (c @ W[p + "uv"].T).view(T, H, dv)
    s = (torch.einsum("ihd,jhd->hij", qn, k) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (i - j >= 0) & (i - j < m["mask"]["size"])
    a = torch.softmax(s.masked_fill(~seen, float("-inf")), -1)
    return torch.einsum("hij,jhd->ihd", a, v).reshape(T, H * dv) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------- Mamba-2
def causal_conv(x, w, b):
    T, taps = x.shape[0], w.shape[1]
    xp = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x], 0)
    y = b.expand(T, -1).clone()
    for k in range(taps):
        y = y + xp[k:k + T] * w[:, k]
    return y


def state_space(x, B, C, dt, A_log, D):
    """x [T, H, P], B / C [T, G, N], dt [T, H] after softplus; one token after another."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = x.new_zeros(H, N, P)
    out = []
    group = torch.arange(H) // (H // G)
    for t in range(T):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][group][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, C[t][group]) + D[:, None] * x[t])
    return torch.stack(out)


def mamba2(W, p, m, eps, h):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    t = h @ W[p + "in"].T
    z, xbc, dt = t[:, :inner], t[:, inner:2 * inner + 2 * G * N], t[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = xbc[:, :inner].reshape(T, H, P), xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    y = state_space(x, B, C, softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"]).reshape(T, inner)
    y = (y * silu(z)).reshape(T, m["norm_groups"], -1)
    return (unit_rms(y, eps).reshape(T, inner) * W[p + "norm"]) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------- feed-forward, side input
def dense_ff(W, p, h):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def token_side(W, p, dim, i, eps, x, tokens):
    e = W["side.embed"][tokens][:, i * dim:(i + 1) * dim]
    y = (gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T
    return unit_rms(y, eps) * W[p + "side.norm"]


# ------------------------------------------------------------------------------------------- the model
def model(cfg, W, tokens, residuals=None):
    """Logits [T, vocab] of one sequence; ``residuals`` (a list) receives the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(tokens).long()
    positions = torch.arange(len(tokens))
    x = W["embed"][tokens]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = dynamic_tanh(x, W[p + "norm1"], W[p + "norm1.b"], W[p + "norm1.alpha"])
        if layer["type"] == "mamba2":
            y = mamba2(W, p + "mix.", m, eps, h)
        else:
            j = m.get("kv_from")
            if j is None:
                kept[i] = latent_of(W, p + "mix.", m, eps, h, positions)
            y = latent_attention(W, p + "mix.", m, eps, h, positions, *kept[i if j is None else j])
        if layer["mlp"] is not None:
            y = y + dense_ff(W, p + "mlp.", h)
        x = x + y
        x = x + token_side(W, p, cfg["token_side"]["dim"], i, eps, x, tokens)
        if residuals is not None:
            residuals.append(x)
    return dynamic_tanh(x, W["final.norm"], W["final.norm.b"], W["final.norm.alpha"]) @ W["head"].T


# ------------------------------------------------------------------------------------------- checkpoints for tests
def tensor_shapes(cfg):
    """name -> shape of every tensor of a checkpoint with this configuration."""
    V, H, L, sd = cfg["vocab"], cfg["width"], len(cfg["layers"]), cfg["token_side"]["dim"]
    out = {"embed": (V, H), "side.embed": (V, L * sd), "head": (V, H)}

    def norm(name):
        out.update({name: (H,), name + ".b": (H,), name + ".alpha": ()})

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        norm(p + "norm1")
        if layer["type"] == "mamba2":
            inner, bc = m["heads"] * m["vdim"], 2 * m["groups"] * m["state"]
            out.update({p + "mix.in": (2 * inner + bc + m["heads"], H), p + "mix.conv": (inner + bc, m["conv"]), p + "mix.conv.b": (inner + bc,),
                        p + "mix.dt_bias": (m["heads"],), p + "mix.A_log": (m["heads"],), p + "mix.D": (m["heads"],),
                        p + "mix.norm": (inner,), p + "mix.o": (H, inner)})
        else:
            h = m["heads"]
            out.update({p + "mix.dq": (m["q_rank"], H), p + "mix.dq.norm": (m["q_rank"],), p + "mix.uq": (h * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                        p + "mix.uk": (h * m["dim"], m["kv_rank"]), p + "mix.uv": (h * m["vdim"], m["kv_rank"]), p + "mix.o": (H, h * m["vdim"])})
            if m.get("kv_from") is None:
                out.update({p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], H), p + "mix.dkv.norm": (m["kv_rank"],)})
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            out.update({p + "mlp.gate": (f, H), p + "mlp.up": (f, H), p + "mlp.down": (H, f)})
        out.update({p + "side.gate": (sd, H), p + "side.proj": (H, sd), p + "side.norm": (H,)})
    return out


def random_weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random bf16-representable weights with scales at which every branch matters."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "alpha":
            t = torch.rand(shape, generator=g) * 0.5 + 0.6
        elif leaf in ("norm", "norm1"):
            t = 1 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "b":
            t = 0.1 * torch.randn(shape, generator=g)
        elif leaf == "dt_bias":
            t = torch.rand(shape, generator=g) * 3 - 4
        elif leaf == "A_log":
            t = torch.rand(shape, generator=g) * 2 - 0.5
        elif leaf == "D":
            t = 0.5 + torch.rand(shape, generator=g)
        elif leaf == "conv":
            t = torch.randn(shape, generator=g) / shape[1] ** 0.5
        elif leaf == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
        W[name] = t.to(torch.bfloat16).to(dtype)
    return W


def write_checkpoint(path, cfg, W):
    """``config.json`` + ``model.safetensors`` (bf16) under ``path``."""
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    head, blobs, at = {}, [], 0
    for name, t in W.items():
        raw = t.to(torch.bfloat16).contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    js = json.dumps(head).encode()
    (path / "model.safetensors").write_bytes(struct.pack("<Q", len(js)) + js + b"".join(blobs))
    return path
