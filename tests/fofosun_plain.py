"""Plain, slow statement of the Fofosun decoder in 64-bit PyTorch: one function per mechanism, one token or one query at a
time, no cache, no batching, no kernels. It shares no code with the package; the tests compare the package with it.

A model is ``(cfg, W)``: the configuration dictionary and a dictionary of weight tensors under their checkpoint names.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------ element-wise pieces
def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def unit_rms(x, eps):
    """x over its root mean square, along the last axis; eps under the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def dyt_norm(x, w, b, alpha):
    """Dynamic Tanh: squashes every element by itself, then scales and shifts it."""
    return torch.tanh(alpha * x) * w + b


def poly_norm(z, coef, eps):
    c1, c2, c3, c0 = (coef[i] for i in range(4))
    return c1 * unit_rms(z, eps) + c2 * unit_rms(z * z, eps) + c3 * unit_rms(z * z * z, eps) + c0


def rotate_pairs(v, pos, base, dims):
    """Turns neighbours (2i, 2i + 1), i < dims / 2, of the vector(s) ``v`` [..., n] by pos * base^(-2i / dims)."""
    out = v.clone()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        c, s = math.cos(a), math.sin(a)
        x, y = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = x * c - y * s
        out[..., 2 * i + 1] = y * c + x * s
    return out


# ------------------------------------------------------------------------------------------ mixers: x [tokens, width] -> same
def hgrn2(W, p, m, h, eps, state=None):
    """The forget gate f of a channel keeps that row of the state; its complement 1 - f writes the value."""
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = silu(h @ W[p + "q"].T).reshape(T, H, dk)
    v = (h @ W[p + "v"].T).reshape(T, H, dv)
    low = W[p + "lower"]
    f = (low + (1.0 - low) * sigmoid(h @ W[p + "f"].T + W[p + "f.b"])).reshape(T, H, dk)
    S = torch.zeros(H, dk, dv, dtype=h.dtype) if state is None else state
    rows = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hkv,hk->hv", S, q[t]))
    o = rms_norm(torch.stack(rows), W[p + "norm"], eps)
    return o.reshape(T, H * dv) @ W[p + "o"].T


def lightning(W, p, m, h, eps, state=None):
    """One constant decay per head; the heads are normed together and gated."""
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = silu(h @ W[p + "q"].T).reshape(T, H, dk)
    k = silu(h @ W[p + "k"].T).reshape(T, H, dk)
    v = silu(h @ W[p + "v"].T).reshape(T, H, dv)
    decay = torch.tensor(m["decay"], dtype=h.dtype).reshape(H, 1, 1)
    S = torch.zeros(H, dk, dv, dtype=h.dtype) if state is None else state
    rows = []
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hkv,hk->hv", S, q[t]))
    o = rms_norm(torch.stack(rows).reshape(T, H * dv), W[p + "norm"], eps) * sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def latent_attention(W, p, m, h, eps):
    """Softmax attention whose keys and values come from one low-rank latent per token plus one rotated key part."""
    H, d, r, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    base = m["rot"]["base"]
    cq = rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps)
    q = (cq @ W[p + "uq"].T).reshape(T, H, d + r)
    kv = h @ W[p + "dkv"].T
    c = rms_norm(kv[:, :kr], W[p + "dkv.norm"], eps)
    k_un = (c @ W[p + "uk"].T).reshape(T, H, d)
    v = (c @ W[p + "uv"].T).reshape(T, H, dv)
    q_rot = torch.stack([rotate_pairs(q[t, :, d:], t, base, r) for t in range(T)])
    k_rot = torch.stack([rotate_pairs(kv[t, kr:], t, base, r) for t in range(T)])
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        s = torch.einsum("hd,jhd->hj", q[t, :, :d], k_un[: t + 1]) + torch.einsum("hd,jd->hj", q_rot[t], k_rot[: t + 1])
        s = s * m["scale"]
        s = torch.exp(s - s.max(dim=-1, keepdim=True).values)
        s = s / s.sum(dim=-1, keepdim=True)
        out[t] = torch.einsum("hj,jhv->hv", s, v[: t + 1])
    return out.reshape(T, H * dv) @ W[p + "o"].T


MIXERS = {"hgrn2": hgrn2, "lightning": lightning, "latent_attention": latent_attention}


def dense_ff(W, p, h, eps):
    return poly_norm(h @ W[p + "up"].T, W[p + "act"], eps) @ W[p + "down"].T


# ------------------------------------------------------------------------------------------ the whole decoder
def norm_at(W, name, x):
    return dyt_norm(x, W[name], W[name + ".b"], W[name + ".alpha"])


def forward(cfg, W, tokens, dtype=F64):
    """-> (logits [tokens, vocab], residual after every layer [layers, tokens, width])."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[layer["type"]](W, p + "mix.", layer["mixer"], norm_at(W, p + "norm1", x), eps)
        x = x + y * W[p + "ls1"]
        if layer["mlp"] is not None:
            x = x + dense_ff(W, p + "mlp.", norm_at(W, p + "norm2", x), eps) * W[p + "ls2"]
        after.append(x)
    return norm_at(W, "final.norm", x) @ W["head"].T, torch.stack(after)
