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


def chunk_mask(T, size, off=0):
    """off: a mistake of so many tokens in where chunks start"""
    i = torch.arange(T)
    return (i[:, None] >= i) & ((i[:, None] + off) // size == (i + off) // size)


def distance_bias(T, r1, r2):
    """[H, T, T], what is taken off the scores (i ≥ j)"""
    d = (torch.arange(T)[:, None] - torch.arange(T)).clamp(min=0).double()
    return r1[:, None, None] * torch.log1p(r2[:, None, None] * d)


def attend(q, k, v, r1, r2, m, off=0):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] (normed) → [T, H · vdim]"""
    T, H = len(q), m["heads"]
    seen, off = chunk_mask(T, m["mask"]["size"], off), distance_bias(T, r1, r2)
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


# ---- configurations and weights of the tests ---------------------------------------------------------------------------------------

def delta(heads=6, kv_heads=3, dim=24, vdim=40, conv=4, decay_rank=10, gate_rank=7):
    return {"conv": conv, "decay_rank": decay_rank, "dim": dim, "gate_rank": gate_rank, "heads": heads, "kv_heads": kv_heads, "vdim": vdim}


def latent(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=56, q_rank=48, scale=None, base=700.0):
    return {"dim": dim, "heads": heads, "kv_rank": kv_rank, "q_rank": q_rank, "rot": {"base": base, "dims": rot_dim}, "rot_dim": rot_dim,
            "scale": scale if scale is not None else 1.2 / math.sqrt(dim + rot_dim), "vdim": vdim}


def attn(heads=6, kv_heads=2, dim=16, vdim=24, size=20, scale=None, kv_from=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": size}, "scale": scale if scale is not None else 1.3 / math.sqrt(dim), "vdim": vdim}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def layer(mixer, ff=72):
    kind = "channel_delta" if "conv" in mixer else "latent_attention" if "kv_rank" in mixer else "attention"
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def make_config(layers, width=64, vocab=131, eps=1e-5, mult=0.6, softcap=12.0, side=16):
    return {"architecture": "Senadra", "layers": layers, "logit_softcap": softcap, "norm": {"eps": eps}, "residual_mult": mult,
            "token_side": {"dim": side}, "vocab": vocab, "width": width}


def make_weights(cfg, seed=0, gain=1.0):
    """Random weights of every tensor of the checkpoint (bf16-exact values, so every run sees the same numbers)."""
    g = torch.Generator().manual_seed(seed)
    D, n, out = cfg["width"], cfg["token_side"]["dim"], {}

    def lin(name, o, i, k=1.0):
        out[name] = (torch.randn(o, i, generator=g) * k * gain / math.sqrt(i)).bfloat16()

    def vec(name, n, mean=0.0, std=0.2, sign=False):
        t = mean + std * torch.randn(n, generator=g)
        out[name] = (t.abs() if sign else t).bfloat16()

    lin("embed", cfg["vocab"], D, math.sqrt(D))
    lin("side.embed", cfg["vocab"], n * len(cfg["layers"]), math.sqrt(n * len(cfg["layers"])))
    for i, spec in enumerate(cfg["layers"]):
        m, f, p = spec["mixer"], spec["mlp"], f"l{i}."
        vec(p + "norm1", D, 1.0)
        q = p + "mix."
        if spec["type"] == "channel_delta":
            for t, rows in (("q", m["kv_heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["heads"] * m["vdim"])):
                lin(q + t, rows, D, 1.5)
                lin(q + t + ".conv", rows, m["conv"], 1.3)
            lin(q + "b", m["heads"], D, 1.5)
            vec(q + "A_log", m["heads"], -1.5, 1.5)             # heads that forget at once beside heads that remember
            vec(q + "dt_bias", m["heads"] * m["dim"], -1.5, 1.5)
            vec(q + "norm", m["vdim"], 1.0)
            lin(q + "a1", m["decay_rank"], D)
            lin(q + "a2", m["heads"] * m["dim"], m["decay_rank"])
            lin(q + "g1", m["gate_rank"], D)
            lin(q + "g2", m["heads"] * m["vdim"], m["gate_rank"], 1.5)
        elif spec["type"] == "latent_attention":
            lin(q + "dq", m["q_rank"], D)
            vec(q + "dq.norm", m["q_rank"], 1.0)
            lin(q + "uq", m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.5)
            lin(q + "dkv", m["kv_rank"] + m["rot_dim"], D, 1.5)
            vec(q + "dkv.norm", m["kv_rank"], 1.0)
            lin(q + "uk", m["heads"] * m["dim"], m["kv_rank"])
            lin(q + "uv", m["heads"] * m["vdim"], m["kv_rank"])
        else:
            lin(q + "q", m["heads"] * m["dim"], D, 1.5)
            if m.get("kv_from") is None:
                lin(q + "k", m["kv_heads"] * m["dim"], D, 1.5)
                lin(q + "v", m["kv_heads"] * m["vdim"], D)
            vec(q + "r1", m["heads"], 0.6, 0.5, True)
            vec(q + "r2", m["heads"], 0.4, 0.3, True)
        if spec["type"] != "channel_delta":
            lin(q + "g", m["heads"] * m["vdim"], D, 1.5)
        lin(q + "o", D, m["heads"] * m["vdim"])
        if f is not None:
            vec(p + "norm2", D, 1.0)
            lin(p + "mlp.up", f["ff"], D, 1.5)
            lin(p + "mlp.down", D, f["ff"])
            vec(p + "mlp.act", 2, 0.3, 0.7)
        lin(p + "side.gate", n, D, 1.5)
        lin(p + "side.proj", D, n)
        vec(p + "side.norm", D, 0.8)
    vec("final.norm", D, 1.0)
    lin("head", cfg["vocab"], D, 4.0)
    return out
