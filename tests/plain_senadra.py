"""Plain, slow statement of the Senadra decoder: one function per mechanism, whole sequences, float64.

The oracle of the Senadra tests.  It works on a `config.json` dictionary and a dictionary of checkpoint tensors, shares no code
with the package, keeps no cache and no state: logits at a position come from running the sequence up to it.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z):
    return z / 2 * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- gated delta rule with a decay per key channel -------------------------------------------------------------------------------

def short_conv(x, w):
    """x [T, channels], w [channels, taps] (the last column meets the current token) → silu of the causal convolution."""
    T, taps = len(x), w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    y = sum(padded[k:k + T] * w[:, k] for k in range(taps))
    return y * sigmoid(y)


def unit(x):
    return x / torch.sqrt((x ** 2).sum(-1, keepdim=True) + 1e-6)


def log_decays(raw, A_log, dt_bias):
    """raw [T, heads · dim] → [T, heads, dim], the logarithms of the decays."""
    return -torch.exp(A_log)[:, None] * softplus(raw + dt_bias).unflatten(-1, (len(A_log), -1))


def delta_rule(q, k, v, logg, beta):
    """q, k [T, G, K] (unit vectors, q scaled), v [T, H, V], logg [T, H, K], beta [T, H] → [T, H, V], token by token from an empty state."""
    T, H, V = v.shape
    per = H // q.shape[1]
    out = torch.zeros_like(v)
    for h in range(H):
        S = torch.zeros(q.shape[2], V, dtype=v.dtype)
        for t in range(T):
            S = torch.exp(logg[t, h])[:, None] * S
            kt = k[t, h // per]
            S = S + torch.outer(kt, beta[t, h] * (v[t, h] - kt @ S))
            out[t, h] = q[t, h // per] @ S
    return out


def channel_delta(h, W, p, m, eps):
    H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in "qkv")
    q, k = unit(q.unflatten(-1, (G, K))) / math.sqrt(K), unit(k.unflatten(-1, (G, K)))
    logg = log_decays(h @ W[p + "a1"].T @ W[p + "a2"].T, W[p + "A_log"], W[p + "dt_bias"])
    o = delta_rule(q, k, v.unflatten(-1, (H, V)), logg, sigmoid(h @ W[p + "b"].T))
    o = rms(o, eps) * W[p + "norm"] * sigmoid(h @ W[p + "g1"].T @ W[p + "g2"].T).unflatten(-1, (H, V))
    return o.flatten(1) @ W[p + "o"].T


# ---- latent attention -------------------------------------------------------------------------------------------------------------

def rotate(x, base):
    """x [T, ..., dims], pairs (2i, 2i + 1) turned by position · base^(−2i/dims)."""
    T, d = len(x), x.shape[-1]
    f = torch.tensor([base ** (-2 * i / d) for i in range(d // 2)], dtype=x.dtype)
    a = (torch.arange(T, dtype=x.dtype)[:, None] * f).reshape([T] + [1] * (x.dim() - 2) + [d // 2])
    u, v = x[..., ::2], x[..., 1::2]
    return torch.stack([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()], -1).flatten(-2)


def latent_of(h, W, p, m, eps):
    """(latent [T, rank], shared rotated key part [T, rot_dim] before its rotation)"""
    c, r = (h @ W[p + "dkv"].T).split([m["kv_rank"], m["rot_dim"]], -1)
    return rms(c, eps) * W[p + "dkv.norm"], r


def latent_heads(q, c, kr, W, p, m):
    """q [T, H, dim + rot_dim] and kr [T, rot_dim] before rotation, c the latents → [T, H · vdim]"""
    H, d = m["heads"], m["dim"]
    base = m["rot"]["base"]
    qr, kr = rotate(q[..., d:], base), rotate(kr, base)
    k, v = (c @ W[p + "uk"].T).unflatten(-1, (H, d)), (c @ W[p + "uv"].T).unflatten(-1, (H, m["vdim"]))
    out = []
    for h in range(H):
        e = (q[:, h, :d] @ k[:, h].T + qr[:, h] @ kr.T) * m["scale"]
        e = e.masked_fill(torch.ones_like(e, dtype=torch.bool).triu(1), -math.inf)
        out.append(torch.softmax(e, -1) @ v[:, h])
    return torch.cat(out, -1)


def latent_attention(h, W, p, m, eps):
    q = rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"] @ W[p + "uq"].T
    o = latent_heads(q.unflatten(-1, (m["heads"], -1)), *latent_of(h, W, p, m, eps), W, p, m)
    return o * sigmoid(h @ W[p + "g"].T) @ W[p + "o"].T


# ---- attention inside chunks, with a distance bias ----------------------------------------------------------------------------------

def keys_values(h, W, p, m, eps):
    """([T, G, dim], [T, G, vdim]), values over their root mean square"""
    return (h @ W[p + "k"].T).unflatten(-1, (m["kv_heads"], m["dim"])), rms((h @ W[p + "v"].T).unflatten(-1, (m["kv_heads"], m["vdim"])), eps)


def chunk_mask(T, size):
    i = torch.arange(T)
    return (i[:, None] >= i) & (i[:, None] // size == i // size)


def distance_bias(T, r1, r2):
    """[H, T, T], what is taken off the scores (i ≥ j)"""
    d = (torch.arange(T)[:, None] - torch.arange(T)).clamp(min=0).double()
    return r1[:, None, None] * torch.log1p(r2[:, None, None] * d)


def attend(q, k, v, r1, r2, m):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] (normed) → [T, H · vdim]"""
    T, H = len(q), m["heads"]
    seen, off = chunk_mask(T, m["mask"]["size"]), distance_bias(T, r1, r2)
    out = []
    for h in range(H):
        g = h // (H // m["kv_heads"])
        e = q[:, h] @ k[:, g].T * m["scale"] - off[h]
        out.append(torch.softmax(e.masked_fill(~seen, -math.inf), -1) @ v[:, g])
    return torch.cat(out, -1)


def attention(h, W, p, m, kv):
    o = attend((h @ W[p + "q"].T).unflatten(-1, (m["heads"], m["dim"])), *kv, W[p + "r1"], W[p + "r2"], m)
    return o * sigmoid(h @ W[p + "g"].T) @ W[p + "o"].T


# ---- feed-forward, per-layer token input --------------------------------------------------------------------------------------------

def xielu(z, act):
    a, b = softplus(act[0]), softplus(act[1])
    neg = z.clamp(max=0)
    return z / 2 + torch.where(z > 0, a * z ** 2, (0.5 + b) * (torch.expm1(neg) - neg))


def feed_forward(h, W, p):
    return xielu(h @ W[p + "up"].T, W[p + "act"]) @ W[p + "down"].T


def side_input(x, rows, W, p, eps):
    """x the residual, rows [T, dim] the layer's part of the token vectors → what is added (before the residual's factor)"""
    y = gelu_tanh(x @ W[p + "gate"].T) * rows @ W[p + "proj"].T
    return rms(y, eps) * W[p + "norm"]


@torch.no_grad()
def run(cfg, W, tokens, layers=None):
    """Logits of every position; `layers` (a list) receives the residual after every layer."""
    W = {k: v.double() for k, v in W.items()}
    eps, mult, n = cfg["norm"]["eps"], cfg["residual_mult"], cfg["token_side"]["dim"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"][tokens]
    kept: dict = {}
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}."
        h = rms(x, eps) * W[p + "norm1"]
        if spec["type"] == "channel_delta":
            y = channel_delta(h, W, p + "mix.", m, eps)
        elif spec["type"] == "latent_attention":
            y = latent_attention(h, W, p + "mix.", m, eps)
        else:
            if m.get("kv_from") is None:
                kept[i] = keys_values(h, W, p + "mix.", m, eps)
            y = attention(h, W, p + "mix.", m, kept[i if m.get("kv_from") is None else m["kv_from"]])
        x = x + mult * y
        if spec["mlp"] is not None:
            x = x + mult * feed_forward(rms(x, eps) * W[p + "norm2"], W, p + "mlp.")
        x = x + mult * side_input(x, W["side.embed"][tokens][:, i * n:(i + 1) * n], W, p + "side.", eps)
        if layers is not None:
            layers.append(x)
    z = rms(x, eps) * W["final.norm"] @ W["head"].T
    return cfg["logit_softcap"] * torch.tanh(z / cfg["logit_softcap"])
