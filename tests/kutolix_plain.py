"""Plain, slow statement of the Kutolix decoder in 64-bit PyTorch: one function per mechanism, one query at a time, no cache, no
batching, no kernels. It shares no code with the package; the tests compare the package with it.

A model is ``(cfg, W)``: the configuration dictionary and a dictionary of weight tensors under their checkpoint names.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------ pieces
def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return over_rms(x, eps) * w


def frequencies(rot):
    """-> (turn rate of every pair, factor on its sine and cosine). With ``scaling``: slow pairs turn ``factor`` times slower, fast
    ones as they are, a ramp in between."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def where(turns):                          # the pair that makes this many turns over the original length
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / sc["factor"] * r + v * (1.0 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(v, p, rot, neighbours):
    """The first rot.dims entries of v [..., width] turned by the angles of position p; pairs are neighbouring entries, or an entry and
    the one half the rotated width behind it."""
    f, mul = frequencies(rot)
    n = rot["dims"] // 2
    out = v.clone()
    for i in range(n):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + n)
        c, s = math.cos(p * f[i]) * mul, math.sin(p * f[i]) * mul
        out[..., a] = v[..., a] * c - v[..., b] * s
        out[..., b] = v[..., b] * c + v[..., a] * s
    return out


def first_visible(t, mask):
    """First position that position t sees."""
    return max(0, t - mask["size"] + 1) if mask else 0


# ------------------------------------------------------------------------------------------ mixers: h [tokens, width] -> same
def windowed_attention(W, p, m, h, eps):
    """Grouped-query softmax attention over a window: queries and keys turned, then brought to unit root mean square; one more term
    in every denominator; the result gated element by element."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k = (h @ W[p + "q"].T).reshape(T, H, d), (h @ W[p + "k"].T).reshape(T, G, d)
    v = (h @ W[p + "v"].T).reshape(T, G, dv)
    q = over_rms(torch.stack([rotate(q[t], t, m["rot"], False) for t in range(T)]), eps)
    k = over_rms(torch.stack([rotate(k[t], t, m["rot"], False) for t in range(T)]), eps)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        a = first_visible(t, m["mask"])
        for n in range(H):
            g = n // (H // G)
            s = k[a: t + 1, g] @ q[t, n] * m["scale"]
            top = max(s.max().item(), W[p + "sink"][n].item())
            e = torch.exp(s - top)
            out[t, n] = (e @ v[a: t + 1, g]) / (e.sum() + torch.exp(W[p + "sink"][n] - top))
    return (out.reshape(T, H * dv) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def latent_attention(W, p, m, h, eps):
    """Attention whose keys and values are made from a short latent per token, beside one turned key part that all heads share."""
    H, d, r, dv, kr = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    q = (h @ W[p + "q"].T).reshape(T, H, d + r)
    low = h @ W[p + "dkv"].T
    c = rms_norm(low[:, :kr], W[p + "dkv.norm"], eps)
    kr_ = torch.stack([rotate(low[t, kr:], t, m["rot"], True) for t in range(T)])
    qr = torch.stack([rotate(q[t, :, d:], t, m["rot"], True) for t in range(T)])
    k, v = (c @ W[p + "uk"].T).reshape(T, H, d), (c @ W[p + "uv"].T).reshape(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        a = first_visible(t, m["mask"])
        for n in range(H):
            s = (k[a: t + 1, n] @ q[t, n, :d] + kr_[a: t + 1] @ qr[t, n]) * m["scale"]
            e = torch.exp(s - s.max())
            out[t, n] = (e @ v[a: t + 1, n]) / e.sum()
    return out.reshape(T, H * dv) @ W[p + "o"].T


MIXERS = {"attention": windowed_attention, "latent_attention": latent_attention}


# ------------------------------------------------------------------------------------------ feed-forwards
def dense_ff(W, p, m, h):
    g = h @ W[p + "gate"].T
    return (g * sigmoid(g) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def clamped_ff(W, p, m, h):
    """One expert."""
    g = torch.clamp(h @ W[p + "gate"].T, max=m["limit"])
    u = torch.clamp(h @ W[p + "up"].T, min=-m["limit"], max=m["limit"])
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def choose(z, m):
    """Router logits of one token -> [(expert, weight)]: softmax over all; the best experts of the groups with the best members."""
    e = torch.exp(z - z.max())
    s = (e / e.sum()).tolist()
    groups = m.get("groups") or {"count": 1, "keep": 1}
    per = len(s) // groups["count"]
    best = sorted(range(groups["count"]), key=lambda g: -max(s[g * per:(g + 1) * per]))[: groups["keep"]]
    open_ = [i for i in range(len(s)) if i // per in best]
    return [(i, s[i]) for i in sorted(open_, key=lambda i: -s[i])[: m["top"]]]


def routed_ff(W, p, m, h):
    z = h @ W[p + "router"].T
    rows = []
    for t in range(h.shape[0]):
        y = torch.zeros_like(h[t])
        for e, w in choose(z[t], m["router"]):
            y = y + w * clamped_ff(W, f"{p}e{e}.", m["expert"], h[t])
        rows.append(y)
    return torch.stack(rows)


FEED_FORWARDS = {"dense": dense_ff, "moe": routed_ff}


# ------------------------------------------------------------------------------------------ the whole decoder
def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


def forward(cfg, W, tokens, dtype=F64):
    """-> (logits [tokens, vocab], the residual after every layer [layers, tokens, width])."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + m * rms_norm(MIXERS[layer["type"]](W, p + "mix.", layer["mixer"], x, eps), W[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = x + m * rms_norm(FEED_FORWARDS[layer["mlp"]["kind"]](W, p + "mlp.", layer["mlp"], x), W[p + "norm2"], eps)
        after.append(x)
    return soft_cap(rms_norm(x, W["final.norm"], eps) @ W["embed"].T, cfg["logit_softcap"]), torch.stack(after)
