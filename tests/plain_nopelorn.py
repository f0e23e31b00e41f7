"""Plain, slow statement of the Nopelorn decoder: one function per mechanism, whole sequences, float64 unless told otherwise.

The oracle of the Nopelorn tests.  It works on a `config.json` dictionary and a dictionary of checkpoint tensors, shares no code
with the package, keeps no cache and no state between calls: logits at a position come from running the sequence up to it.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z / (1 + torch.exp(-z))


def embed(tokens, W, spec):
    """Token rows plus rows of the hashed bigram table; the first token takes the table's last row."""
    x = W["embed"][tokens].clone()
    big = (spec or {}).get("bigram")
    if big:
        table = W["bigram"]
        for t, tok in enumerate(tokens.tolist()):
            row = big["buckets"] if t == 0 else (int(tokens[t - 1]) * big["mul_prev"] + tok * big["mul_cur"]) % big["buckets"]
            x[t] += table[row]
    return x


def yarn_frequencies(rot):
    """(frequency per pair, factor of cos and sin)."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim(turns):
        return n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(dim(sc["fast"])), 0), min(math.ceil(dim(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, rot):
    """x [T, ..., n]: token t at position t; pairs are (2i, 2i + 1)."""
    f, mag = yarn_frequencies(rot)
    y = x.clone()
    for t in range(x.shape[0]):
        for i, fi in enumerate(f):
            c, s = math.cos(t * fi) * mag, math.sin(t * fi) * mag
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            y[t, ..., 2 * i] = u * c - v * s
            y[t, ..., 2 * i + 1] = v * c + u * s
    return y


def visible(T, window):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = i >= j
    return ok & (i - j < window) if window else ok


def softmax_sink(scores, sink):
    """scores [H, T, S] (−inf where masked), sink [H]: a bare exp(sink) in the denominator."""
    m = torch.maximum(scores.amax(-1), sink[:, None])
    e = torch.exp(scores - m[..., None])
    return e / (e.sum(-1) + torch.exp(sink[:, None] - m))[..., None]


def latent_of(h, W, pre, m, eps):
    kv = h @ W[pre + "dkv"].T
    c = rms(kv[:, : m["kv_rank"]], eps) * W[pre + "dkv.norm"]
    return c, rotate(kv[:, m["kv_rank"]:], m["rot"])


def latent_attention(h, W, pre, m, eps, latent):
    T, H, dn, dr, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ W[pre + "q"].T).view(T, H, dn + dr)
    qn, qr = q[..., :dn], rotate(q[..., dn:], m["rot"])
    c, kr = latent
    k = (c @ W[pre + "uk"].T).view(T, H, dn)
    v = (c @ W[pre + "uv"].T).view(T, H, dv)
    s = (torch.einsum("thd,shd->hts", qn, k) + torch.einsum("thd,sd->hts", qr, kr)) * m["scale"]
    s = s.masked_fill(~visible(T, (m.get("mask") or {}).get("size"))[None], -math.inf)
    p = softmax_sink(s, W[pre + "sink"])
    return torch.einsum("hts,shd->thd", p, v).reshape(T, H * dv) @ W[pre + "o"].T


def lightning_states(q, k, v, decay):
    """q, k [T, H, dk], v [T, H, dv] → outputs [T, H, dv], one token after another."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out)


def lightning(h, W, pre, m, eps):
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (silu(h @ W[pre + n].T).view(T, H, dk) for n in "qk")
    v = silu(h @ W[pre + "v"].T).view(T, H, dv)
    o = lightning_states(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)).reshape(T, H * dv)
    o = rms(o, eps) * W[pre + "norm"] / (1 + torch.exp(-(h @ W[pre + "g"].T)))
    return o @ W[pre + "o"].T


def clamped_ff(h, W, pre, m):
    lim = m["limit"]
    g = (h @ W[pre + "gate"].T).clamp(max=lim)
    u = (h @ W[pre + "up"].T).clamp(-lim, lim)
    return (g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ W[pre + "down"].T


def run(cfg, weights, tokens, dtype=torch.float64, layers=None):
    """Logits [T, vocab]; `layers` (a list) collects the residual stream after every layer."""
    W = {n: t.to(dtype) if t.is_floating_point() else t for n, t in weights.items()}
    tokens = torch.as_tensor(tokens)
    eps = cfg["norm"]["eps"]
    x = embed(tokens, W, cfg.get("embedding"))
    latents = {}
    for i, spec in enumerate(cfg["layers"]):
        m, pre = spec["mixer"], f"l{i}.mix."
        if spec["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                latents[i] = latent_of(x, W, pre, m, eps)
            y = latent_attention(x, W, pre, m, eps, latents[i if src is None else src])
        else:
            y = lightning(x, W, pre, m, eps)
        x = x + rms(y, eps) * W[f"l{i}.norm1"] * W[f"l{i}.ls1"]
        if spec["mlp"] is not None:
            y = clamped_ff(x, W, f"l{i}.mlp.", spec["mlp"])
            x = x + rms(y, eps) * W[f"l{i}.norm2"] * W[f"l{i}.ls2"]
        if layers is not None:
            layers.append(x.clone())
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T


# ---- small random models for the tests ------------------------------------------------------------------------------------

def latent_spec(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=32, window=19, scale=None, base=5000.0, kv_from=None,
                factor=4.0, original=64, fast=16.0, slow=2.0, ff=96, limit=1.5):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
         "scale": scale if scale is not None else 1.3 / math.sqrt(dim + rot_dim),
         "rot": {"base": base, "dims": rot_dim, "scaling": {"factor": factor, "original": original, "fast": fast, "slow": slow}},
         "mask": {"size": window}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def lightning_spec(heads=2, dim=16, vdim=24, decay=None, ff=96, limit=1.5):
    decay = decay or [0.55 + 0.44 * (h + 1) / (heads + 1) for h in range(heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def make_config(layers, width=64, vocab=131, buckets=97, mul_prev=13, mul_cur=5, eps=1e-5):
    return {"architecture": "Nopelorn", "embedding": {"bigram": {"buckets": buckets, "mul_cur": mul_cur, "mul_prev": mul_prev}},
            "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def make_weights(cfg, seed=0, dtype=torch.bfloat16, gain=1.0):
    """Random weights of every tensor of the checkpoint (bf16-exact values, so every run sees the same numbers)."""
    g = torch.Generator().manual_seed(seed)
    D, V = cfg["width"], cfg["vocab"]
    out = {}

    def lin(name, o, i):
        out[name] = (torch.randn(o, i, generator=g) * gain / math.sqrt(i)).to(dtype)

    def vec(name, n, mean=1.0, std=0.2):
        out[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)

    out["embed"] = torch.randn(V, D, generator=g).to(dtype)
    if cfg.get("embedding", {}).get("bigram"):
        out["bigram"] = (0.7 * torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, D, generator=g)).to(dtype)
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}.mix."
        H = m["heads"]
        if spec["type"] == "latent_attention":
            lin(p + "q", H * (m["dim"] + m["rot_dim"]), D)
            if m.get("kv_from") is None:
                lin(p + "dkv", m["kv_rank"] + m["rot_dim"], D)
                vec(p + "dkv.norm", m["kv_rank"])
            lin(p + "uk", H * m["dim"], m["kv_rank"])
            lin(p + "uv", H * m["vdim"], m["kv_rank"])
            vec(p + "sink", H, 0.5, 1.0)
            lin(p + "o", D, H * m["vdim"])
        else:
            lin(p + "q", H * m["dim"], D)
            lin(p + "k", H * m["dim"], D)
            lin(p + "v", H * m["vdim"], D)
            lin(p + "g", H * m["vdim"], D)
            vec(p + "norm", H * m["vdim"])
            lin(p + "o", D, H * m["vdim"])
        vec(f"l{i}.norm1", D)
        vec(f"l{i}.ls1", D, 0.6)
        if spec["mlp"] is not None:
            F = spec["mlp"]["ff"]
            lin(f"l{i}.mlp.gate", F, D)
            lin(f"l{i}.mlp.up", F, D)
            lin(f"l{i}.mlp.down", D, F)
            vec(f"l{i}.norm2", D)
            vec(f"l{i}.ls2", D, 0.6)
    vec("final.norm", D)
    lin("head", V, D)
    return out
