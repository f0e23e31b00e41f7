"""Plain, slow statement of the Ronupel decoder: one function per mechanism, whole sequences, float64.

The oracle of the Ronupel tests.  It works on a `config.json` dictionary and a dictionary of checkpoint tensors, shares no code
with the package, keeps no cache: logits at a position come from running the sequence up to it.
"""
from __future__ import annotations

import math

import torch


def rms(x, w, eps):
    return w * x / torch.sqrt((x ** 2).mean(-1, keepdim=True) + eps)


def angles(positions, rot):
    """[T, dims / 2]"""
    per_step = [rot["base"] ** (-2 * i / rot["dims"]) / (rot["scaling"]["factor"] if rot.get("scaling") else 1) for i in range(rot["dims"] // 2)]
    return positions.double()[:, None] * torch.tensor(per_step, dtype=torch.float64)


def rotate(x, positions, rot, back=False):
    """x [T, heads, dim]: neighbours 2i and 2i + 1 of the first `dims` dimensions turn together."""
    if not rot:
        return x
    a = angles(positions, rot)[:, None]
    z = torch.view_as_complex(x[..., : rot["dims"]].unflatten(-1, (-1, 2)).contiguous())
    z = z * torch.polar(torch.ones_like(a), -a if back else a)
    return torch.cat([torch.view_as_real(z).flatten(-2), x[..., rot["dims"]:]], -1)


def prepared(rows, w, heads, positions, m, eps):
    """Queries or keys of all heads: normed over the whole row, then split and rotated."""
    return rotate(rms(rows, w, eps).unflatten(-1, (heads, m["dim"])), positions, m.get("rot"))


def visible(i: int, j: int, mask) -> bool:
    if j > i:
        return False
    return not mask or i - j < mask["size"] or j < mask.get("keep_first", 0)


def attend(q, k, v, sink, m):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] of a whole sequence → [T, H · vdim]"""
    T, H = q.shape[:2]
    sees = torch.tensor([[visible(i, j, m.get("mask")) for j in range(T)] for i in range(T)])
    out = []
    for h in range(H):
        g = h // (H // m["kv_heads"])
        e = q[:, h] @ k[:, g].T * m["scale"]
        e = torch.where(sees, e, torch.full_like(e, -math.inf))
        top = torch.maximum(e.max(1).values, sink[h])[:, None]
        num = torch.exp(e - top)
        out.append(num @ v[:, g] / (num.sum(1, keepdim=True) + torch.exp(sink[h] - top)))
    return torch.cat(out, 1)


def attention(h, W, p, m, eps):
    pos = torch.arange(len(h))
    q = prepared(h @ W[p + "q"].T, W[p + "q.norm"], m["heads"], pos, m, eps)
    k = prepared(h @ W[p + "k"].T, W[p + "k.norm"], m["kv_heads"], pos, m, eps)
    v = (h @ W[p + "v"].T).unflatten(-1, (m["kv_heads"], m["vdim"]))
    return attend(q, k, v, W[p + "sink"], m) @ W[p + "o"].T


def glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g / (1 + torch.exp(-1.702 * g)) * (u + 1)


def expert(h, W, p, limit):
    return glu(h @ W[p + ".gate"].T, h @ W[p + ".up"].T, limit) @ W[p + ".down"].T


def choose(z, top):
    """(indices, weights) of the `top` largest logits of every row."""
    order = torch.argsort(z, dim=-1, descending=True, stable=True)[:, :top]
    e = torch.exp(z.gather(1, order) - z.max(-1, keepdim=True).values)
    return order, e / e.sum(-1, keepdim=True)


def mixture(h, W, p, f):
    idx, w = choose(h @ W[p + "router"].T + W[p + "router.b"], f["router"]["top"])
    rows = []
    for t in range(len(h)):
        y = sum(w[t, j] * expert(h[t], W, f"{p}e{int(e)}", f["expert"]["limit"]) for j, e in enumerate(idx[t]))
        rows.append(y)
    y = torch.stack(rows)
    return y + expert(h, W, p + "shared", f["shared"]["limit"]) if f.get("shared") else y


def order_of_runs(cfg):
    """(layer, embedding output added before it) of every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    out = [(i, False) for i in range(loop["start"])]
    for p in range(loop["times"]):
        for i in range(loop["start"], loop["stop"]):
            out.append((i, p > 0 and i == loop["start"]))
    return out + [(i, False) for i in range(loop["stop"], n)]


@torch.no_grad()
def run(cfg, W, tokens, layers=None):
    """Logits of every position; `layers` (a list) receives the residual after every layer run."""
    W = {k: v.double() for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    first = x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, again in order_of_runs(cfg):
        if again:
            x = x + first
        spec = cfg["layers"][i]
        h = rms(x, W[f"l{i}.norm1"], eps)
        y = attention(h, W, f"l{i}.mix.", spec["mixer"], eps)
        if spec["mlp"] is not None:
            y = y + mixture(h, W, f"l{i}.mlp.", spec["mlp"])
        x = x + y
        if layers is not None:
            layers.append(x)
    return rms(x, W["final.norm"], eps) @ W["embed"].T


# ---- configurations and weights of the tests ---------------------------------------------------------------------------------

def mixer_spec(heads=6, kv_heads=2, dim=24, vdim=40, window=19, keep=5, rot=16, base=3000.0, factor=3.0, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.4 / math.sqrt(dim)}
    if rot:
        m["rot"] = {"base": base, "dims": rot, "scaling": {"factor": factor}}
        if factor is None:
            del m["rot"]["scaling"]
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    return m


def layer_spec(experts=5, top=2, ff=56, limit=1.3, shared=72, shared_limit=2.1, **mixer):
    mlp = None
    if experts:
        mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
        if shared:
            mlp["shared"] = {"ff": shared, "limit": shared_limit}
    return {"type": "attention", "mixer": mixer_spec(**mixer), "mlp": mlp}


def make_config(layers, width=64, vocab=131, loop=None, eps=1e-5):
    cfg = {"architecture": "Ronupel", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def make_weights(cfg, seed=0, gain=1.0):
    """Random weights of every tensor of the checkpoint (bf16-exact values, so every run sees the same numbers)."""
    g = torch.Generator().manual_seed(seed)
    D, out = cfg["width"], {}

    def lin(name, o, i, k=1.0):
        out[name] = (torch.randn(o, i, generator=g) * k * gain / math.sqrt(i)).bfloat16()

    def vec(name, n, mean=1.0, std=0.2):
        out[name] = (mean + std * torch.randn(n, generator=g)).bfloat16()

    def ff(name, n):
        lin(name + ".gate", n, D, 1.5)
        lin(name + ".up", n, D, 1.5)
        lin(name + ".down", D, n)

    out["embed"] = torch.randn(cfg["vocab"], D, generator=g).bfloat16()
    for i, spec in enumerate(cfg["layers"]):
        m, f, p = spec["mixer"], spec["mlp"], f"l{i}."
        vec(p + "norm1", D)
        lin(p + "mix.q", m["heads"] * m["dim"], D)
        lin(p + "mix.k", m["kv_heads"] * m["dim"], D)
        lin(p + "mix.v", m["kv_heads"] * m["vdim"], D)
        vec(p + "mix.q.norm", m["heads"] * m["dim"])
        vec(p + "mix.k.norm", m["kv_heads"] * m["dim"])
        vec(p + "mix.sink", m["heads"], 0.5, 1.0)
        lin(p + "mix.o", D, m["heads"] * m["vdim"])
        if f is not None:
            for e in range(f["router"]["experts"]):
                ff(f"{p}mlp.e{e}", f["expert"]["ff"])
            lin(p + "mlp.router", f["router"]["experts"], D, 2.0)
            vec(p + "mlp.router.b", f["router"]["experts"], 0.0, 1.0)
            if f.get("shared"):
                ff(p + "mlp.shared", f["shared"]["ff"])
    vec("final.norm", D)
    return out
