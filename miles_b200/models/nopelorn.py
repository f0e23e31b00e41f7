"""Nopelorn: `config.json` ⇄ `LayeredConfig`, checkpoint names ⇄ this package's names.

A Nopelorn model lists its layers one by one; each is latent attention (sliding window, softmax sink, YaRN rotary, optionally
on another layer's latents) or decayed linear attention, with a clamped gated feed-forward or none.  Checkpoint tensors are
called `l<i>.mix.*`, `l<i>.mlp.*`, `l<i>.norm1/2`, `l<i>.ls1/2`, `embed`, `bigram`, `final.norm`, `head`; here the projections
of one input are stacked (`mix.w_in`, `mix.w_ukv`, `mlp.w13`).
"""
from __future__ import annotations

import re

import torch

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

_TOP = {"embed": "embed", "bigram": "bigram", "final.norm": "norm", "head": "lm_head"}


def is_checkpoint(names) -> bool:
    return any(re.match(r"l\d+\.", n) or n in ("final.norm", "head") for n in names)


def _stacks(spec: LayerSpec) -> dict[str, list[tuple[str, int]]]:
    """Our stacked tensor → the checkpoint tensors it holds, in order, with their row counts."""
    m = spec.mixer
    if isinstance(m, LatentSpec):
        w_in = [("mix.q", m.heads * (m.dim + m.rot_dim))] + ([("mix.dkv", m.kv_rank + m.rot_dim)] if m.kv_from is None else [])
        out = {"mix.w_in": w_in, "mix.w_ukv": [("mix.uk", m.heads * m.dim), ("mix.uv", m.heads * m.vdim)]}
    else:
        out = {"mix.w_in": [("mix.q", m.heads * m.dim), ("mix.k", m.heads * m.dim), ("mix.v", m.heads * m.vdim), ("mix.g", m.heads * m.vdim)]}
    if spec.mlp is not None:
        out["mlp.w13"] = [("mlp.gate", spec.mlp.ff), ("mlp.up", spec.mlp.ff)]
    return out


def _singles(spec: LayerSpec) -> dict[str, str]:
    m = spec.mixer
    out = {"norm1": "norm1", "ls1": "ls1", "mix.wo": "mix.o"}
    if isinstance(m, LatentSpec):
        if m.kv_from is None:
            out["mix.kv_norm"] = "mix.dkv.norm"
        if m.sink:
            out["mix.sink"] = "mix.sink"
    else:
        out["mix.norm"] = "mix.norm"
    if spec.mlp is not None:
        out.update({"norm2": "norm2", "ls2": "ls2", "mlp.w2": "mlp.down"})
    return out


def place(name: str, cfg: LayeredConfig) -> tuple[str, int, int | None] | None:
    """Where a checkpoint tensor goes: (our tensor, first row, rows; None: all of it).  None for a name that is none of the design's."""
    if name in _TOP:
        return _TOP[name], 0, None
    m = re.match(r"l(\d+)\.(.+)", name)
    if not m or int(m.group(1)) >= cfg.num_layers:
        return None
    i, rest = int(m.group(1)), m.group(2)
    for ours, parts in _stacks(cfg.layer_specs[i]).items():
        at = 0
        for n, rows in parts:
            if n == rest:
                return f"layers.{i}.{ours}", at, rows
            at += rows
    for ours, n in _singles(cfg.layer_specs[i]).items():
        if n == rest:
            return f"layers.{i}.{ours}", 0, None
    return None


def load_into(params: dict, named, cfg: LayeredConfig) -> set:
    """Copy checkpoint tensors (any subset: the parts of a stack may come apart) into the model's parameters.  Returns the
    parameters of which every row was given."""
    rows: dict[str, int] = {}
    for name, t in named:
        where = place(name, cfg)
        if where is None:
            continue
        ours, at, n = where
        p = params[ours].data
        dst = p if n is None else p[at:at + n]
        assert tuple(t.shape) == tuple(dst.shape), f"{name}: got {tuple(t.shape)}, the configuration says {tuple(dst.shape)}"
        dst.copy_(t)
        rows[ours] = rows.get(ours, 0) + dst.shape[0]
    return {n for n, r in rows.items() if r >= params[n].shape[0]}


def from_checkpoint(named: dict[str, torch.Tensor], cfg: LayeredConfig) -> dict[str, torch.Tensor]:
    out = {ours: named[n] for n, ours in _TOP.items() if n in named}
    for i, s in enumerate(cfg.layer_specs):
        for ours, parts in _stacks(s).items():
            if all(f"l{i}.{n}" in named for n, _ in parts):
                ts = [named[f"l{i}.{n}"] for n, _ in parts]
                for t, (n, rows) in zip(ts, parts):
                    assert t.shape[0] == rows, f"l{i}.{n}: {t.shape[0]} rows, the configuration says {rows}"
                out[f"layers.{i}.{ours}"] = torch.cat(ts, 0)
        for ours, n in _singles(s).items():
            if f"l{i}.{n}" in named:
                out[f"layers.{i}.{ours}"] = named[f"l{i}.{n}"]
    return out


def to_checkpoint(name: str, tensor: torch.Tensor, cfg: LayeredConfig) -> list[tuple[str, torch.Tensor]]:
    """One tensor of ours → the checkpoint's tensors."""
    inv = {v: k for k, v in _TOP.items()}
    if name in inv:
        return [(inv[name], tensor)]
    m = re.match(r"layers\.(\d+)\.(.+)", name)
    i, rest = int(m.group(1)), m.group(2)
    stacks = _stacks(cfg.layer_specs[i])
    if rest in stacks:
        parts = stacks[rest]
        return [(f"l{i}.{n}", t) for (n, _), t in zip(parts, tensor.split([r for _, r in parts], 0))]
    return [(f"l{i}.{_singles(cfg.layer_specs[i])[rest]}", tensor)]


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
