"""Plain, slow statement of the Vozirax decoder: one function per mechanism, whole sequences, float64.

The oracle of the Vozirax tests.  It works on a `config.json` dictionary and a dictionary of checkpoint tensors, shares no code
with the package, keeps no cache and no state: logits at a position come from running the sequence up to it.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps)


def place_vectors(T: int, width: int):
    """[T, width] sines at the even, cosines at the odd entries of a pair that shares its frequency."""
    out = torch.zeros(T, width, dtype=torch.float64)
    p = torch.arange(T, dtype=torch.float64)
    for c in range(width):
        a = p * 10000.0 ** (-(c - c % 2) / width)
        out[:, c] = torch.cos(a) if c % 2 else torch.sin(a)
    return out


# ---- state-space mixer ---------------------------------------------------------------------------------------------------------

def short_conv(x, w, b):
    """x [T, channels], w [channels, taps] (the last column meets the current token) → silu of the causal convolution."""
    T, taps = len(x), w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    y = b + sum(padded[k:k + T] * w[:, k] for k in range(taps))
    return y * torch.sigmoid(y)


def step_sizes(raw, bias):
    z = raw + bias
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def recurrence(x, B, C, dt, A_log, D):
    """x [T, H, V], B and C [T, G, N], dt [T, H] → [T, H, V], token by token from an empty state."""
    T, H, V = x.shape
    per = H // B.shape[1]
    y = torch.zeros_like(x)
    for h in range(H):
        S = torch.zeros(B.shape[2], V, dtype=x.dtype)
        for t in range(T):
            S = S * torch.exp(-torch.exp(A_log[h]) * dt[t, h]) + dt[t, h] * torch.outer(B[t, h // per], x[t, h])
            y[t, h] = C[t, h // per] @ S + D[h] * x[t, h]
    return y


def part_norm(y, z, w, parts, eps):
    """Gate first, then every part by its own root mean square."""
    g = y * z * torch.sigmoid(z)
    return rms(g.unflatten(-1, (parts, -1)), eps).flatten(-2) * w


def state_space(h, W, p, m, eps):
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    z, xbc, dt = (h @ W[p + "in"].T).split([H * V, H * V + 2 * G * N, H], -1)
    x, B, C = short_conv(xbc, W[p + "conv"], W[p + "conv.b"]).split([H * V, G * N, G * N], -1)
    y = recurrence(x.unflatten(-1, (H, V)), B.unflatten(-1, (G, N)), C.unflatten(-1, (G, N)), step_sizes(dt, W[p + "dt_bias"]),
                   W[p + "A_log"], W[p + "D"])
    return part_norm(y.flatten(1), z, W[p + "norm"], m["norm_groups"], eps) @ W[p + "o"].T


# ---- differential attention ----------------------------------------------------------------------------------------------------

def temperature(T: int, q_temp):
    """[T] factor on the queries of every position."""
    if not q_temp:
        return torch.ones(T, dtype=torch.float64)
    return torch.tensor([1 + q_temp["coef"] * math.log((p + 1) // q_temp["every"] + 1) for p in range(T)], dtype=torch.float64)


def keys_values(h, W, p, m, eps):
    """([T, G, 2, dim], [T, G, vdim])"""
    k = rms((h @ W[p + "k"].T).unflatten(-1, (m["kv_heads"], 2, m["dim"])), eps) * W[p + "k.norm"]
    return k, (h @ W[p + "v"].T).unflatten(-1, (m["kv_heads"], m["vdim"]))


def one_map(q, k, v, scale):
    e = q @ k.T * scale
    e = e.masked_fill(torch.ones_like(e, dtype=torch.bool).triu(1), -math.inf)
    return torch.softmax(e, -1) @ v


def mix_weight(W, p, diff):
    return torch.exp((W[p + "lq1"] * W[p + "lk1"]).sum()) - torch.exp((W[p + "lq2"] * W[p + "lk2"]).sum()) + diff


def difference(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1 - diff)


def attend(q, k, v, gate, lam, m, eps):
    """q [T, H, 2, dim] (normed, tempered), k [T, G, 2, dim], v [T, G, vdim], gate [T, H] (before the sigmoid) → [T, H · vdim]"""
    out = []
    for h in range(m["heads"]):
        g = h // (m["heads"] // m["kv_heads"])
        a1, a2 = (one_map(q[:, h, i], k[:, g, i], v[:, g], m["scale"]) for i in (0, 1))
        out.append(difference(a1, a2, lam, m["diff"], eps) * torch.sigmoid(gate[:, h, None]))
    return torch.cat(out, -1)


def queries(rows, w, m, eps):
    q = rms(rows.unflatten(-1, (m["heads"], 2, m["dim"])), eps) * w
    return q * temperature(len(q), m.get("q_temp"))[:, None, None, None]


def attention(h, W, p, m, eps, kv):
    q = queries(h @ W[p + "q"].T, W[p + "q.norm"], m, eps)
    return attend(q, *kv, h @ W[p + "g"].T, mix_weight(W, p, m["diff"]), m, eps) @ W[p + "o"].T


# ---- feed-forward ----------------------------------------------------------------------------------------------------------------

def dense(h, W, p):
    g = h @ W[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def expert(h, W, p):
    return torch.clamp(h @ W[p + ".up"].T, min=0) ** 2 @ W[p + ".down"].T


def choose(z, correction, r):
    """(indices, weights) of every row of router logits."""
    s = torch.sigmoid(z)
    c = s + correction
    n = (r.get("groups") or {}).get("count", 1)
    keep = (r.get("groups") or {}).get("keep", 1)
    size = z.shape[1] // n
    idx, wts = [], []
    for t in range(len(z)):
        worth = [sum(sorted(c[t, g * size:(g + 1) * size].tolist(), reverse=True)[:2]) for g in range(n)]
        good = sorted(range(n), key=lambda g: (-worth[g], g))[:keep]
        open_ = [e for g in good for e in range(g * size, (g + 1) * size)]
        best = sorted(open_, key=lambda e: (-float(c[t, e]), e))[: r["top"]]
        idx.append(best)
        w = s[t, best]
        wts.append(w / (w.sum() + 1e-20) * r["scale"])
    return torch.tensor(idx), torch.stack(wts)


def mixture(h, W, p, f):
    idx, w = choose(h @ W[p + "router"].T, W[p + "correction"], f["router"])
    return torch.stack([sum(w[t, j] * expert(h[t], W, f"{p}e{int(e)}") for j, e in enumerate(idx[t])) for t in range(len(h))])


@torch.no_grad()
def run(cfg, W, tokens, layers=None):
    """Logits of every position; `layers` (a list) receives the residual after every layer."""
    W = {k: v.double() for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = x + place_vectors(len(x), cfg["width"])
    kept: dict = {}
    for i, spec in enumerate(cfg["layers"]):
        m, f, p = spec["mixer"], spec["mlp"], f"l{i}."
        h = rms(x, eps) * (1 + W[p + "norm1"])
        if spec["type"] == "mamba2":
            y = state_space(h, W, p + "mix.", m, eps)
        else:
            if m.get("kv_from") is None:
                kept[i] = keys_values(h, W, p + "mix.", m, eps)
            y = attention(h, W, p + "mix.", m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        y = y * W[p + "ls1"]
        if f is not None:
            h = rms(x, eps) * (1 + W[p + "norm2"])
            y = y + W[p + "ls2"] * (dense(h, W, p + "mlp.") if f["kind"] == "dense" else mixture(h, W, p + "mlp.", f))
        x = x + y
        if layers is not None:
            layers.append(x)
    return (rms(x, eps) * (1 + W["final.norm"])) @ W["head"].T * cfg["logit_scale"]


# ---- configurations and weights of the tests ---------------------------------------------------------------------------------

def ssm(heads=6, vdim=24, state=40, groups=2, taps=4, norm_groups=3):
    return {"conv": taps, "groups": groups, "heads": heads, "norm_groups": norm_groups, "state": state, "vdim": vdim}


def attn(heads=6, kv_heads=3, dim=16, vdim=40, diff=0.35, scale=None, coef=0.4, every=9, kv_from=None):
    m = {"diff": diff, "dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale if scale is not None else 1.3 / math.sqrt(dim), "vdim": vdim}
    if coef is not None:
        m["q_temp"] = {"coef": coef, "every": every}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def ff(n=72):
    return {"kind": "dense", "ff": n}


def moe(experts=8, top=3, n=40, count=4, keep=2, scale=1.7):
    r = {"experts": experts, "scale": scale, "top": top}
    if count:
        r["groups"] = {"count": count, "keep": keep}
    return {"kind": "moe", "expert": {"ff": n}, "router": r}


def layer(mixer, mlp):
    return {"type": "mamba2" if "state" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def make_config(layers, width=64, vocab=131, eps=1e-5, logit_scale=0.7):
    return {"architecture": "Vozirax", "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def make_weights(cfg, seed=0, gain=1.0, apart=False):
    """Random weights of every tensor of the checkpoint (bf16-exact values, so every run sees the same numbers).  `apart`: corrections that
    decide the choice of groups and experts whatever the scores (no close calls for 16-bit runs; the weights of the choice still differ by token)."""
    g = torch.Generator().manual_seed(seed)
    D, out = cfg["width"], {}

    def lin(name, o, i, k=1.0):
        out[name] = (torch.randn(o, i, generator=g) * k * gain / math.sqrt(i)).bfloat16()

    def vec(name, n, mean=0.0, std=0.2):
        out[name] = (mean + std * torch.randn(n, generator=g)).bfloat16()

    lin("embed", cfg["vocab"], D, math.sqrt(D))
    for i, spec in enumerate(cfg["layers"]):
        m, f, p = spec["mixer"], spec["mlp"], f"l{i}."
        vec(p + "norm1", D)
        vec(p + "ls1", D, 0.8)
        if spec["type"] == "mamba2":
            inner, H, n = m["heads"] * m["vdim"], m["heads"], m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"]
            lin(p + "mix.in", inner + n + H, D, 1.5)
            lin(p + "mix.conv", n, m["conv"], 1.2)
            vec(p + "mix.conv.b", n)
            vec(p + "mix.dt_bias", H, -1.0, 1.0)
            vec(p + "mix.A_log", H, -1.0, 1.5)          # heads that forget at once beside heads that remember
            vec(p + "mix.D", H, 0.5, 0.5)
            vec(p + "mix.norm", inner, 1.0)
            lin(p + "mix.o", D, inner)
        else:
            lin(p + "mix.q", m["heads"] * 2 * m["dim"], D)
            if m.get("kv_from") is None:
                lin(p + "mix.k", m["kv_heads"] * 2 * m["dim"], D)
                lin(p + "mix.v", m["kv_heads"] * m["vdim"], D)
                vec(p + "mix.k.norm", m["dim"], 1.0)
            vec(p + "mix.q.norm", m["dim"], 1.0)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                vec(p + "mix." + n, m["dim"], 0.0, 0.3)
            lin(p + "mix.g", m["heads"], D)
            lin(p + "mix.o", D, m["heads"] * m["vdim"])
        if f is None:
            continue
        vec(p + "norm2", D)
        vec(p + "ls2", D, 0.8)
        if f["kind"] == "dense":
            lin(p + "mlp.gate", f["ff"], D, 1.5)
            lin(p + "mlp.up", f["ff"], D, 1.5)
            lin(p + "mlp.down", D, f["ff"])
        else:
            for e in range(f["router"]["experts"]):
                lin(f"{p}mlp.e{e}.up", f["expert"]["ff"], D, 1.2)
                lin(f"{p}mlp.e{e}.down", D, f["expert"]["ff"])
            lin(p + "mlp.router", f["router"]["experts"], D, 2.0)
            vec(p + "mlp.correction", f["router"]["experts"], -0.3, 0.4)   # some choice scores are negative
            if apart:
                out[p + "mlp.correction"] = (4.0 * 1.9 ** torch.randperm(f["router"]["experts"], generator=g) - 9.0).bfloat16()
    vec("final.norm", D)
    lin("head", cfg["vocab"], D, 2.0)
    return out
