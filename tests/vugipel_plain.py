"""Plain, slow statement of the Vugipel decoder in 64-bit PyTorch: one function per mechanism, one token or one query at a time, no
cache, no batching, no kernels. It shares no code with the package; the tests compare the package with it.

A model is ``(cfg, W)``: the configuration dictionary and a dictionary of weight tensors under their checkpoint names.
"""
from __future__ import annotations

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------ pieces
def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return over_rms(x, eps) * (1.0 + w)


def turn_pairs(v, positions, base, dims):
    """Row t of v [rows, heads, width]: neighbouring entries (2 i, 2 i + 1) of the first ``dims`` turned by positions[t] base^(-2 i / dims)."""
    a = torch.tensor([[p * base ** (-2.0 * i / dims) for i in range(dims // 2)] for p in positions], dtype=F64)[:, None]
    c, s = torch.cos(a).to(v.dtype), torch.sin(a).to(v.dtype)
    out = v.clone()
    x, y = v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2] = x * c - y * s
    out[..., 1:dims:2] = y * c + x * s
    return out


def visible(t, mask):
    """Positions that position t sees: the first ``keep_first``, and those less than ``size`` back."""
    return [j for j in range(t + 1) if not mask or t - j < mask["size"] or j < mask.get("keep_first", 0)]


def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


# ------------------------------------------------------------------------------------------ mixers: h [tokens, width] -> same
def candidate(u):
    """What a gated recurrence takes in: positive, bending into a line at zero."""
    return torch.where(u >= 0, u + 0.5, sigmoid(u))


def min_gru(W, p, m, h, eps, state=None):
    """A recurrence per channel whose gate and candidate read the token alone; the result gated by a third projection."""
    z = sigmoid(h @ W[p + "z"].T + W[p + "z.b"])
    c = candidate(h @ W[p + "x"].T + W[p + "x.b"])
    S = torch.zeros(m["width"], dtype=h.dtype) if state is None else state
    rows = []
    for t in range(h.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        rows.append(S)
    return (torch.stack(rows) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def rotated_value_attention(W, p, m, h, eps):
    """Grouped-query softmax attention over a window and the first tokens: projections with biases; queries and keys normed, then
    turned; values turned by their own position and the result turned back by the query's; scores times a number per head,
    softly capped."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, rot = h.shape[0], m["rot"]
    proj = lambda n, heads, w: (h @ W[p + n].T + W[p + n + ".b"]).reshape(T, heads, w)
    q = over_rms(proj("q", H, d), eps) * W[p + "q.norm"]
    k = over_rms(proj("k", G, d), eps) * W[p + "k.norm"]
    v = proj("v", G, dv)
    q, k = (turn_pairs(x, range(T), rot["base"], rot["dims"]) for x in (q, k))
    v = turn_pairs(v, range(T), rot["base"], dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        j = visible(t, m["mask"])
        for n in range(H):
            g = n // (H // G)
            s = soft_cap(k[j, g] @ q[t, n] * m["scale"] * W[p + "temp"][n], m["softcap"])
            e = torch.exp(s - s.max())
            out[t, n] = (e @ v[j, g]) / e.sum()
    out = turn_pairs(out, [-t for t in range(T)], rot["base"], dv)
    return out.reshape(T, H * dv) @ W[p + "o"].T + W[p + "o.b"]


def retention(W, p, m, h, eps, state=None):
    """Per head a matrix that fades by a constant and to which k v^T is added; read with q, brought to unit root mean square, gated."""
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (h @ W[p + "q"].T).reshape(T, H, dk)
    k = (h @ W[p + "k"].T).reshape(T, H, dk) * dk ** -0.5
    v = (h @ W[p + "v"].T).reshape(T, H, dv)
    decay = torch.tensor(m["decay"], dtype=h.dtype)
    S = torch.zeros(H, dk, dv, dtype=h.dtype) if state is None else state
    rows = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        rows.append(torch.einsum("hkv,hk->hv", S, q[t]))
    o = over_rms(torch.stack(rows), eps).reshape(T, H * dv)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel(W, p, m, h, eps):
    left = rotated_value_attention(W, p + "left.", m["left"], h, eps)
    right = retention(W, p + "right.", m["right"], h, eps)
    return m["left_scale"] * left + m["right_scale"] * right


MIXERS = {"mingru": min_gru, "parallel": parallel}


# ------------------------------------------------------------------------------------------ feed-forward
def expert(W, p, h):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def choose(z, m):
    """Router logits of one token -> [(expert, weight)]: the largest sigmoids, as they are."""
    s = sigmoid(z).tolist()
    return [(i, s[i]) for i in sorted(range(len(s)), key=lambda i: -s[i])[: m["top"]]]


def routed_ff(W, p, m, h):
    """An expert's weight multiplies what the expert reads."""
    z = h @ W[p + "router"].T
    rows = []
    for t in range(h.shape[0]):
        y = torch.zeros_like(h[t])
        for e, w in choose(z[t], m["router"]):
            y = y + expert(W, f"{p}e{e}.", w * h[t])
        rows.append(y)
    return torch.stack(rows)


# ------------------------------------------------------------------------------------------ the whole decoder
def forward(cfg, W, tokens, dtype=F64):
    """-> (logits [tokens, vocab], the residual after every layer [layers, tokens, width])."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](W, p + "mix.", layer["mixer"], centred_norm(x, W[p + "norm1"], eps), eps)
        if layer["mlp"] is not None:
            x = x + routed_ff(W, p + "mlp.", layer["mlp"], centred_norm(x, W[p + "norm2"], eps))
        after.append(x)
    return centred_norm(x, W["final.norm"], eps) @ W["head"].T, torch.stack(after)
