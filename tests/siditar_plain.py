"""Plain, slow statement of the Siditar decoder in 64-bit PyTorch: one function per mechanism, one token or one query at a time, no
cache, no batching, no kernels. It shares no code with the package; the tests compare the package with it.

A model is ``(cfg, W)``: the configuration dictionary and a dictionary of weight tensors under their checkpoint names.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------ pieces
def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, w, eps):
    """x over its root mean square along the last axis, times w."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def layer_norm(x, w, eps):
    """Mean taken off, over the root of the mean squared deviation, times w; no shift."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w


def position_vector(p, width):
    """Sine and cosine of p over wavelengths that grow geometrically with the column pair."""
    out = torch.zeros(width, dtype=F64)
    for c in range(width):
        i = c // 2
        a = p * 10000.0 ** (-2.0 * i / width)
        out[c] = math.sin(a) if c % 2 == 0 else math.cos(a)
    return out


def distance_bucket(n, B, D):
    """Row of the bias table for a key n tokens back: exact up to half the table, then logarithmic up to distance D."""
    half = B // 2
    if n < half:
        return n
    return min(B - 1, half + math.floor(math.log(n / half) / math.log(D / half) * (B - half)))


def query_temperature(p, coef, every):
    return 1.0 + coef * math.log((p + 1) // every + 1)


# ------------------------------------------------------------------------------------------ mixers: h [tokens, width] -> same
def biased_attention(W, p, m, h, eps):
    """Grouped-query softmax attention: normed queries and keys, position only through a bias by distance and a query
    temperature, one more term in every denominator."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = rms_norm((h @ W[p + "q"].T).reshape(T, H, d), W[p + "q.norm"], eps)
    k = rms_norm((h @ W[p + "k"].T).reshape(T, G, d), W[p + "k.norm"], eps)
    v = (h @ W[p + "v"].T).reshape(T, G, dv)
    rel, sink = W[p + "rel"], W[p + "sink"]
    rows = [distance_bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)]
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        temp = query_temperature(t, m["q_temp"]["coef"], m["q_temp"]["every"])
        back = torch.tensor([rows[t - j] for j in range(t + 1)])
        for a in range(H):
            g = a // (H // G)
            s = (k[: t + 1, g] @ (q[t, a] * temp)) * m["scale"] + rel[back, a]
            top = max(s.max().item(), sink[a].item())
            e = torch.exp(s - top)
            out[t, a] = (e @ v[: t + 1, g]) / (e.sum() + torch.exp(sink[a] - top))
    return out.reshape(T, H * dv) @ W[p + "o"].T


def gated_linear_attention(W, p, m, h, eps, state=None):
    """Per head a matrix whose rows fade with a decay of their own and to which k v^T is added; read with q."""
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (h @ W[p + "q"].T).reshape(T, H, dk) * dk ** -0.5
    k = (h @ W[p + "k"].T).reshape(T, H, dk)
    v = (h @ W[p + "v"].T).reshape(T, H, dv)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = (sigmoid(z) ** (1.0 / m["tau"])).reshape(T, H, dk)
    S = torch.zeros(H, dk, dv, dtype=h.dtype) if state is None else state
    rows = []
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hkv,hk->hv", S, q[t]))
    o = rms_norm(torch.stack(rows), W[p + "norm"], eps).reshape(T, H * dv)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel(W, p, m, h, eps):
    left = biased_attention(W, p + "left.", m["left"], h, eps)
    right = gated_linear_attention(W, p + "right.", m["right"], h, eps)
    return m["left_scale"] * left + m["right_scale"] * right


MIXERS = {"parallel": parallel}


def clamped_ff(W, p, m, h):
    g = torch.clamp(h @ W[p + "gate"].T, max=m["limit"])
    u = torch.clamp(h @ W[p + "up"].T, min=-m["limit"], max=m["limit"])
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


# ------------------------------------------------------------------------------------------ residual streams
def read_streams(x, w):
    """x [streams, tokens, width] -> the weighted sum a sublayer reads."""
    return sum(w[s] * x[s] for s in range(x.shape[0]))


def write_streams(x, mix, out, y):
    """Every stream anew from all old ones (mix[from, to]) and the sublayer's result."""
    n = x.shape[0]
    return torch.stack([sum(mix[s, t] * x[s] for s in range(n)) + out[t] * y for t in range(n)])


def layer_runs(n, loop):
    """Indices of the layers in the order they run."""
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


# ------------------------------------------------------------------------------------------ the whole decoder
def forward(cfg, W, tokens, dtype=F64):
    """-> (logits [tokens, vocab], sum of the streams after every layer run [runs, tokens, width])."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps, width = cfg["norm"]["eps"], cfg["width"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = x + torch.stack([position_vector(p, width) for p in range(len(tokens))]).to(dtype)
    x = torch.stack([x] * cfg["streams"])
    after = []
    for i in layer_runs(len(cfg["layers"]), cfg["loop"]):
        layer, p = cfg["layers"][i], f"l{i}."
        h = layer_norm(read_streams(x, W[p + "hc1.in"]), W[p + "norm1"], eps)
        x = write_streams(x, W[p + "hc1.mix"], W[p + "hc1.out"], MIXERS[layer["type"]](W, p + "mix.", layer["mixer"], h, eps))
        if layer["mlp"] is not None:
            h = layer_norm(read_streams(x, W[p + "hc2.in"]), W[p + "norm2"], eps)
            x = write_streams(x, W[p + "hc2.mix"], W[p + "hc2.out"], clamped_ff(W, p + "mlp.", layer["mlp"], h))
        after.append(x.sum(0))
    return layer_norm(x.sum(0), W["final.norm"], eps) @ W["head"].T, torch.stack(after)
