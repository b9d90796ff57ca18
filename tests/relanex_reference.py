"""Relanex restated from its equations in plain tensor code: whole sequences, dense masks, token loops, one function per
mechanism, float64 on the CPU unless told otherwise.  Shares nothing with the package: it is what the package's kernels
are held to.

Weights are a dict name -> tensor with the checkpoint's names ('embed', 'embed.norm', 'l<i>.norm1' / '.norm1b' /
'.norm2' / '.norm2b' each with '.alpha' and '.b', 'l<i>.mix.*', 'l<i>.mlp.*', 'final.norm', 'head'); the configuration
is config.json's dict.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------------------------ small pieces

def bounded_norm(x, W, name):
    """w * tanh(alpha x) + b, element by element."""
    return torch.tanh(W[name + ".alpha"].reshape(()) * x) * W[name] + W[name + ".b"]


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def stretched_frequencies(rot, dtype=torch.float64):
    """(frequency per pair, factor on cos and sin): low pairs keep their frequency, high pairs are slowed down by
    `factor`, those between the two bounds are blended."""
    dims, base = int(rot["dims"]), float(rot["base"])
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = base ** (-2.0 * i / max(dims, 1))
    sc = rot.get("scaling")
    if not sc:
        return f.to(dtype), 1.0

    def dim_of(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return (f / sc["factor"] * ramp + f * (1 - ramp)).to(dtype), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, pos, rot):
    """Pairs (2i, 2i + 1) of the first rot.dims entries of x [T, heads, D] turned by pos[t] * frequency i."""
    dims = int(rot["dims"])
    f, amp = stretched_frequencies(rot, x.dtype)
    ang = pos.to(x.dtype)[:, None, None] * f
    c, s = torch.cos(ang) * amp, torch.sin(ang) * amp
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def visible(T, window=0):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < window) if window else True)


# ------------------------------------------------------------------------------------------------ mixers

def attention(h, W, p, m, eps):
    """Grouped-query causal softmax attention with biases on q, k and v, rotated q and k, and a learned sink per head."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ W[p + n].T + W[p + n + ".b"] for n in "qkv")
    pos = torch.arange(T)
    q, k, v = rotate(q.view(T, H, D), pos, m["rot"]), rotate(k.view(T, G, D), pos, m["rot"]), v.view(T, G, V)
    out = h.new_zeros(T, H, V)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].T) * m["scale"]
        s = s.masked_fill(~visible(T), float("-inf"))
        s = torch.cat([s, W[p + "sink"][hh].expand(T, 1)], 1)
        out[:, hh] = torch.softmax(s, -1)[:, :T] @ v[:, g]
    return out.reshape(T, H * V) @ W[p + "o"].T


def latent_attention(h, W, p, m, eps):
    """Windowed softmax attention without positions: queries through one normed latent, keys and values through another."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).view(T, H, D)
    c = rms_norm(h @ W[p + "dkv"].T, W[p + "dkv.norm"], eps)
    k, v = (c @ W[p + "uk"].T).view(T, H, D), (c @ W[p + "uv"].T).view(T, H, V)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"]
    s = s.masked_fill(~visible(T, m["mask"]["size"] if m.get("mask") else 0), float("-inf"))
    return torch.einsum("hij,jhv->ihv", torch.softmax(s, -1), v).reshape(T, H * V) @ W[p + "o"].T


def log_sigmoid(z):
    return torch.minimum(z, torch.zeros_like(z)) - torch.log1p(torch.exp(-z.abs()))


def mlstm_cell(q, k, v, i, f):
    """q (scaled), k [T, H, D], v [T, H, V], log gates i, f [T, H] -> o [T, H, V]: the stabilised recurrence token by token."""
    T, H, D = q.shape
    S, n, m = q.new_zeros(H, D, v.shape[-1]), q.new_zeros(H, D), q.new_zeros(H)
    out = torch.empty_like(v)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return out


def mlstm(h, W, p, m, eps):
    T, H, D, V, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    q, k, v = (h @ W[p + "q"].T).view(T, H, D) * D ** -0.5, (h @ W[p + "k"].T).view(T, H, D), (h @ W[p + "v"].T).view(T, H, V)
    i = cap * torch.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap))
    o = rms_norm(mlstm_cell(q, k, v, i, f), 1.0, eps).reshape(T, H * V)
    return (o * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


MIXERS = {"attention": attention, "latent_attention": latent_attention, "mlstm": mlstm}


# ------------------------------------------------------------------------------------------------ the model

def silu(z):
    return z * torch.sigmoid(z)


def feed_forward(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def layer_runs(cfg):
    """[(layer index, whether the embedding output is added first)] in running order."""
    n, loop = len(cfg["layers"]), cfg.get("loop") or {}
    start, stop, times = int(loop.get("start", 0)), int(loop.get("stop", 0)), int(loop.get("times", 1))
    if stop <= start:
        return [(i, False) for i in range(n)]
    inner = [(i, t > 0 and i == start) for t in range(times) for i in range(start, stop)]
    return [(i, False) for i in range(start)] + inner + [(i, False) for i in range(stop, n)]


def layer(x, W, cfg, i):
    L, eps, mult, p = cfg["layers"][i], float(cfg["norm"]["eps"]), float(cfg["residual_mult"]), f"l{i}."
    y = MIXERS[L["type"]](bounded_norm(x, W, p + "norm1"), W, p + "mix.", L["mixer"], eps)
    x = x + mult * bounded_norm(y, W, p + "norm1b")
    if L.get("mlp"):
        x = x + mult * bounded_norm(feed_forward(bounded_norm(x, W, p + "norm2"), W, p + "mlp."), W, p + "norm2b")
    return x


def forward(tokens, W, cfg, dtype=torch.float64, collect=None):
    """tokens [T] -> logits [T, vocab]; `collect`, if a list, receives the stream after every layer run."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in W.items()}
    first = bounded_norm(W["embed"][torch.as_tensor(tokens).long()], W, "embed.norm")
    x = first
    for i, again in layer_runs(cfg):
        x = layer(x + first if again else x, W, cfg, i)
        if collect is not None:
            collect.append(x.clone())
    return bounded_norm(x, W, "final.norm") @ W["head"].T
