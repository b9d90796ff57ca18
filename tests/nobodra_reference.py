"""Nobodra restated from its equations in plain tensor code: whole sequences, dense masks, token loops, one function per
mechanism, float64 on the CPU unless told otherwise.  Shares nothing with the package: it is what the package's
kernels are held to.

Weights are a dict name -> tensor with the checkpoint's names ('embed', 'l<i>.norm1' / '.norm2', 'l<i>.mix.*',
'l<i>.mlp.*', 'final.norm', 'head'); the configuration is config.json's dict.
"""
from __future__ import annotations

import torch


# ------------------------------------------------------------------------------------------------ small pieces

def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_plain(x, w, eps):
    return unit_rms(x, eps) * w


def rms_around_one(x, w, eps):
    """The gain is stored as its distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def causal_conv(u, w):
    """u [T, C], w [C, taps]: y[t] = sum_j w[:, j] u[t - taps + 1 + j], zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] = y[back:] + u[:T - back] * w[:, j]
    return y


def rotate_halves(x, base, dims):
    """x [T, heads, D], row t at position t: entries i and i + dims/2 (i < dims/2) are turned by t * base^(-2i/dims)."""
    half = dims // 2
    y = x.clone()
    for i in range(half):
        f = torch.tensor(float(base), dtype=x.dtype) ** (-2.0 * i / dims)
        a = torch.arange(x.shape[0], dtype=x.dtype) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i] = u * c - v * s
        y[:, :, i + half] = v * c + u * s
    return y


def window_mask(T, size):
    """[T, T]: i sees j iff 0 <= i - j < size (size 0: every j <= i)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < size) if size else d >= 0


# ------------------------------------------------------------------------------------------------ mixers

def softmax_attention(q, k, v, scale, size):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]."""
    H, G = q.shape[1], k.shape[1]
    hidden = ~window_mask(q.shape[0], size)
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(hidden, -float("inf"))
        out.append(torch.softmax(s, -1) @ v[:, g])
    return torch.stack(out, 1)


def attention(h, W, p, m, eps):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[p + "q"].T).view(T, H, D)
    raw = (h @ W[p + "k"].T).view(T, G, D)               # the values; normed and turned it is the keys
    q = rms_plain(q, W[p + "q.norm"], eps)
    k = rms_plain(raw, W[p + "k.norm"], eps)
    rot = m.get("rot")
    if rot and rot["dims"]:
        q, k = rotate_halves(q, rot["base"], rot["dims"]), rotate_halves(k, rot["base"], rot["dims"])
    y = softmax_attention(q, k, raw, m["scale"], (m.get("mask") or {}).get("size", 0))
    return y.reshape(T, H * D) @ W[p + "o"].T


def delta_rule(q, k, v, beta, g):
    """q / k [T, G, D], v [T, H, V], beta / g [T, H]; one token after another, state [H, D, V] from zero."""
    T, H, V = v.shape
    rep = H // k.shape[1]
    S = v.new_zeros(H, k.shape[2], V)
    out = []
    for t in range(T):
        kt, qt = k[t].repeat_interleave(rep, 0), q[t].repeat_interleave(rep, 0)
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (S * kt[:, :, None]).sum(1))
        S = S + kt[:, :, None] * u[:, None, :]
        out.append((S * qt[:, :, None]).sum(1))
    return torch.stack(out)


def step_decay(a, A_log, dt_bias):
    return torch.exp(-torch.exp(A_log) * softplus(a + dt_bias))


def delta(h, W, p, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in ("q", "k", "v"))
    q = unit_vector(q.view(T, G, D)) * D ** -0.5
    k = unit_vector(k.view(T, G, D))
    beta = torch.sigmoid(h @ W[p + "b"].T)
    g = step_decay(h @ W[p + "a"].T, W[p + "A_log"], W[p + "dt_bias"])
    o = delta_rule(q, k, v.view(T, H, V), beta, g)
    o = rms_plain(o, W[p + "norm"], eps) * silu(h @ W[p + "g"].T).view(T, H, V)
    return o.reshape(T, H * V) @ W[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward

def route(z, top):
    """z [n] logits of one token -> (chosen ids, weights)."""
    best, ids = torch.topk(z, top)
    return ids, torch.softmax(best, 0)


def expert(h, W, p):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def mixture(h, W, p, mlp):
    z = h @ W[p + "router"].T + W[p + "router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, wts = route(z[t], mlp["router"]["top"])
        for e, w in zip(ids.tolist(), wts):
            out[t] = out[t] + w * expert(h[t], W, f"{p}e{e}.")
    return out


# ------------------------------------------------------------------------------------------------ the model

def forward(tokens, W, cfg, dtype=torch.float64, collect=None):
    """Logits [T, vocab]; `collect`, if a list, receives the stream after every layer."""
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = {"attention": attention, "delta": delta}[layer["type"]]
        x = x + rms_around_one(mixer(x, W, p + "mix.", layer["mixer"], eps), W[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + rms_around_one(mixture(x, W, p + "mlp.", layer["mlp"]), W[p + "norm2"], eps)
        if collect is not None:
            collect.append(x.clone())
    return rms_around_one(x, W["final.norm"], eps) @ W["head"].T
