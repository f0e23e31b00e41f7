"""Nopelorn: `config.json` ⇄ `LayeredConfig`, checkpoint names ⇄ this package's names.

A Nopelorn model lists its layers one by one; each is latent attention (sliding window, softmax sink, YaRN rotary, optionally
on another layer's latents) or decayed linear attention, with a clamped gated feed-forward or none.  Checkpoint tensors are
called `l<i>.mix.*`, `l<i>.mlp.*`, `l<i>.norm1/2`, `l<i>.ls1/2`, `embed`, `bigram`, `final.norm`, `head`; here the projections
of one input are stacked (`mix.w_in`, `mix.w_ukv`, `mlp.w13`).
"""
from __future__ import annotations

from .layered import (BigramSpec, GluSpec, LatentSpec, LayeredConfig, LayerSpec, LinearStateSpec, Rotary, YarnScaling)

ARCHITECTURE = "Nopelorn"


def _mixer(kind: str, m: dict):
    if kind == "latent_attention":
        r = m["rot"]
        sc = r.get("scaling")
        assert r["dims"] == m["rot_dim"], "the rotation covers the rotated part of each head"
        return LatentSpec(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"], scale=m["scale"],
                          rotary=Rotary(r["base"], r["dims"], YarnScaling(sc["factor"], sc["original"], sc["fast"], sc["slow"]) if sc else None),
                          window=(m.get("mask") or {}).get("size") or 0, kv_from=m.get("kv_from"))
    if kind == "lightning":
        return LinearStateSpec(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], decay=tuple(float(d) for d in m["decay"]))
    raise ValueError(f"unknown Nopelorn mixer '{kind}'")


def _mlp(m: dict | None):
    if m is None:
        return None
    if m.get("kind", "dense") != "dense":
        raise ValueError(f"unknown Nopelorn feed-forward '{m['kind']}'")
    return GluSpec(ff=m["ff"], limit=m["limit"])


def from_config(cfg: dict) -> LayeredConfig:
    layers = tuple(LayerSpec(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in cfg["layers"])
    big = (cfg.get("embedding") or {}).get("bigram")
    return LayeredConfig(name=cfg.get("name", "nopelorn"), family="nopelorn", vocab_size=cfg["vocab"], hidden_size=cfg["width"],
                         num_layers=len(layers), num_heads=1, num_kv_heads=1, head_dim=0, ffn_hidden_size=0,
                         rms_eps=cfg["norm"]["eps"], layer_specs=layers,
                         bigram=BigramSpec(big["buckets"], big["mul_prev"], big["mul_cur"]) if big else None)


def to_config(cfg: LayeredConfig) -> dict:
    def layer(s: LayerSpec) -> dict:
        m = s.mixer
        mlp = None if s.mlp is None else {"kind": "dense", "ff": s.mlp.ff, "limit": s.mlp.limit}
        if isinstance(m, LinearStateSpec):
            return {"type": "lightning", "mlp": mlp, "mixer": {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": list(m.decay)}}
        rot: dict = {"base": m.rotary.base, "dims": m.rotary.dims}
        if m.rotary.scaling is not None:
            y = m.rotary.scaling
            rot["scaling"] = {"factor": y.factor, "original": y.original, "fast": y.fast, "slow": y.slow}
        d = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale, "rot": rot}
        if m.window:
            d["mask"] = {"size": m.window}
        if m.kv_from is not None:
            d["kv_from"] = m.kv_from
        return {"type": "latent_attention", "mlp": mlp, "mixer": d}

    out = {"architecture": ARCHITECTURE, "name": cfg.name, "vocab": cfg.vocab_size, "width": cfg.hidden_size,
           "norm": {"eps": cfg.rms_eps}, "layers": [layer(s) for s in cfg.layer_specs]}
    if cfg.bigram is not None:
        b = cfg.bigram
        out["embedding"] = {"bigram": {"buckets": b.buckets, "mul_prev": b.mul_prev, "mul_cur": b.mul_cur}}
    return out


# ---- tensor names -----------------------------------------------------------------------------------------------------

def tensors(cfg: LayeredConfig) -> dict:
    from .designs import Place, rows_of

    out = {"embed": Place("embed"), "final.norm": Place("norm"), "head": Place("lm_head")}
    if cfg.bigram is not None:
        out["bigram"] = Place("bigram")
    for i, s in enumerate(cfg.layer_specs):
        m, l, p = s.mixer, f"l{i}", f"layers.{i}"
        single = {"norm1": "norm1", "ls1": "ls1", "mix.o": "mix.wo"}
        if isinstance(m, LatentSpec):
            out.update(rows_of(f"{p}.mix.w_in", [(f"{l}.mix.q", m.heads * (m.dim + m.rot_dim))]
                               + ([(f"{l}.mix.dkv", m.kv_rank + m.rot_dim)] if m.kv_from is None else [])))
            out.update(rows_of(f"{p}.mix.w_ukv", [(f"{l}.mix.uk", m.heads * m.dim), (f"{l}.mix.uv", m.heads * m.vdim)]))
            if m.kv_from is None:
                single["mix.dkv.norm"] = "mix.kv_norm"
            if m.sink:
                single["mix.sink"] = "mix.sink"
        else:
            out.update(rows_of(f"{p}.mix.w_in", [(f"{l}.mix.q", m.heads * m.dim), (f"{l}.mix.k", m.heads * m.dim),
                                                 (f"{l}.mix.v", m.heads * m.vdim), (f"{l}.mix.g", m.heads * m.vdim)]))
            single["mix.norm"] = "mix.norm"
        if s.mlp is not None:
            out.update(rows_of(f"{p}.mlp.w13", [(f"{l}.mlp.gate", s.mlp.ff), (f"{l}.mlp.up", s.mlp.ff)]))
            single.update({"norm2": "norm2", "ls2": "ls2", "mlp.down": "mlp.w2"})
        out.update({f"{l}.{theirs}": Place(f"{p}.{ours}") for theirs, ours in single.items()})
    return out


_ROT = dict(base=20000.0, dims=16, scaling=YarnScaling(4.0, 256, 24.0, 1.5))

PRESETS = {
    # plumbing-sized model with every kind of layer
    "nopelorn-tiny": LayeredConfig(
        name="nopelorn-tiny", family="nopelorn", vocab_size=512, hidden_size=128, num_layers=4, num_heads=1, num_kv_heads=1, head_dim=0,
        ffn_hidden_size=0, bigram=BigramSpec(257, 19, 3), layer_specs=(
            LayerSpec(LinearStateSpec(4, 16, 32, (0.7, 0.9, 0.97, 0.995)), GluSpec(192, 2.0)),
            LayerSpec(LatentSpec(4, 32, 16, 32, 48, 0.15, Rotary(**_ROT), window=40), GluSpec(192, 2.0)),
            LayerSpec(LinearStateSpec(2, 32, 32, (0.85, 0.98)), None),
            LayerSpec(LatentSpec(2, 48, 16, 64, 48, 0.13, Rotary(**_ROT), window=24, kv_from=1), GluSpec(160, 2.0)))),
    # layer sizes of a mid-sized model: three linear-attention layers per latent-attention layer
    "nopelorn-4B-shape": LayeredConfig(
        name="nopelorn-4B-shape", family="nopelorn", vocab_size=151936, hidden_size=2560, num_layers=36, num_heads=1, num_kv_heads=1,
        head_dim=0, ffn_hidden_size=0, bigram=BigramSpec(65521, 1000003, 8191), layer_specs=tuple(
            LayerSpec(LinearStateSpec(32, 128, 128, tuple(1.0 - 2.0 ** (-2.0 - 6.0 * h / 31) for h in range(32))) if i % 4 != 3 else
                      LatentSpec(32, 128, 64, 128, 512, 0.0722, Rotary(1e6, 64, YarnScaling(8.0, 4096, 32.0, 1.0)), window=1024,
                                 kv_from=i - 4 if i % 8 == 7 else None),
                      GluSpec(9728, 7.0)) for i in range(36))),
}
