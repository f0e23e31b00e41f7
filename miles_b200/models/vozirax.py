"""Vozirax: `config.json` ⇄ `LayeredConfig`, checkpoint names → this package's parameters.

A Vozirax model lists its layers one by one: a state-space mixer or differential attention (which may read an earlier layer's keys and
values) beside a dense feed-forward, a mixture of ungated experts, or none, each behind a norm and before a layer scale of its own.
Positions enter as sinusoidal vectors on the embedding and as a temperature on attention queries.  Checkpoint tensors are called
`l<i>.norm1/2`, `l<i>.ls1/2`, `l<i>.mix.*`, `l<i>.mlp.*`, `embed`, `final.norm`, `head`; here the projections of one input are stacked
along the rows (`mix.w_in`, `mlp.w13`), the four vectors behind the second map's weight form `mix.lvec`, a layer's experts one tensor.
"""
from __future__ import annotations

from ..ops.mixers import Routing
from .layered import (DifferentialSpec, LayeredConfig, LayerSpec, MoeSpec, QueryTemperature, ReluSquareSpec, SsmSpec, plain_glu)

ARCHITECTURE = "Vozirax"
POSITION_BASE = 10000.0


def _mixer(kind: str, m: dict):
    if kind == "mamba2":
        return SsmSpec(heads=m["heads"], vdim=m["vdim"], state=m["state"], groups=m["groups"], conv=m["conv"], norm_groups=m["norm_groups"])
    if kind == "attention":
        t = m.get("q_temp")
        return DifferentialSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], diff=m["diff"],
                                temperature=QueryTemperature(t["coef"], t["every"]) if t else None, kv_from=m.get("kv_from"))
    raise ValueError(f"unknown Vozirax mixer '{kind}'")


def _mlp(m: dict | None):
    if m is None:
        return None
    if m["kind"] == "dense":
        return plain_glu(m["ff"])
    if m["kind"] != "moe":
        raise ValueError(f"unknown Vozirax feed-forward '{m['kind']}'")
    r = m["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    return MoeSpec(experts=r["experts"], top=r["top"], expert=ReluSquareSpec(m["expert"]["ff"]),
                   routing=Routing(groups=g["count"], keep=g["keep"], scale=r["scale"]))


def _config(layers, name: str, vocab: int, width: int, eps: float = 1e-6, logit_scale: float = 1.0) -> LayeredConfig:
    moes = [l.mlp for l in layers if isinstance(l.mlp, MoeSpec)]
    return LayeredConfig(name=name, family="vozirax", vocab_size=vocab, hidden_size=width, num_layers=len(layers), num_heads=1, num_kv_heads=1,
                         head_dim=0, ffn_hidden_size=0, rms_eps=eps, layer_specs=tuple(layers), block="two_norms", norm_shift=1.0,
                         position_base=POSITION_BASE, logit_scale=logit_scale,
                         # what the engine records of the routing: the widest layer's choices
                         num_experts=max((m.experts for m in moes), default=0), moe_topk=max((m.top for m in moes), default=0))


def from_config(cfg: dict) -> LayeredConfig:
    return _config([LayerSpec(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in cfg["layers"]], cfg.get("name", "vozirax"), cfg["vocab"],
                   cfg["width"], cfg["norm"]["eps"], cfg["logit_scale"])


def to_config(cfg: LayeredConfig) -> dict:
    def layer(s: LayerSpec) -> dict:
        m, f = s.mixer, s.mlp
        if isinstance(m, SsmSpec):
            kind, d = "mamba2", {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "conv": m.conv, "norm_groups": m.norm_groups}
        else:
            kind, d = "attention", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "diff": m.diff}
            if m.temperature is not None:
                d["q_temp"] = {"coef": m.temperature.coef, "every": m.temperature.every}
            if m.kv_from is not None:
                d["kv_from"] = m.kv_from
        mlp = None
        if isinstance(f, MoeSpec):
            r = f.routing
            mlp = {"kind": "moe", "expert": {"ff": f.expert.ff},
                   "router": {"experts": f.experts, "top": f.top, "scale": r.scale, "groups": {"count": r.groups, "keep": r.keep}}}
        elif f is not None:
            mlp = {"kind": "dense", "ff": f.ff}
        return {"type": kind, "mixer": d, "mlp": mlp}

    return {"architecture": ARCHITECTURE, "name": cfg.name, "vocab": cfg.vocab_size, "width": cfg.hidden_size, "norm": {"eps": cfg.rms_eps},
            "logit_scale": cfg.logit_scale, "layers": [layer(s) for s in cfg.layer_specs]}


def tensors(cfg: LayeredConfig) -> dict:
    from .designs import Place, rows_of

    out = {"embed": Place("embed"), "final.norm": Place("norm"), "head": Place("lm_head")}
    for i, s in enumerate(cfg.layer_specs):
        m, f, l, p = s.mixer, s.mlp, f"l{i}", f"layers.{i}"
        single = {"norm1": "norm1", "ls1": "ls1", "mix.o": "mix.wo"}
        if isinstance(m, SsmSpec):
            single.update({"mix.in": "mix.w_in", "mix.conv": "mix.conv", "mix.conv.b": "mix.conv_b", "mix.dt_bias": "mix.dt_bias",
                           "mix.A_log": "mix.A_log", "mix.D": "mix.D", "mix.norm": "mix.norm"})
        else:
            rows = [(f"{l}.mix.q", m.heads * 2 * m.dim)]
            if m.kv_from is None:
                rows += [(f"{l}.mix.k", m.kv_heads * 2 * m.dim), (f"{l}.mix.v", m.kv_heads * m.vdim)]
                single["mix.k.norm"] = "mix.k_norm"
            out.update(rows_of(f"{p}.mix.w_in", rows + [(f"{l}.mix.g", m.heads)]))
            single["mix.q.norm"] = "mix.q_norm"
            for k, n in enumerate(("lq1", "lk1", "lq2", "lk2")):
                out[f"{l}.mix.{n}"] = Place(f"{p}.mix.lvec", ((k, k + 1),), True)
        if f is not None:
            single.update({"norm2": "norm2", "ls2": "ls2"})
        if isinstance(f, MoeSpec):
            single.update({"mlp.router": "mlp.router", "mlp.correction": "mlp.correction"})
            for e in range(f.experts):
                out[f"{l}.mlp.e{e}.up"] = Place(f"{p}.mlp.w13", ((e, e + 1),), True)
                out[f"{l}.mlp.e{e}.down"] = Place(f"{p}.mlp.w2", ((e, e + 1),), True)
        elif f is not None:
            out.update(rows_of(f"{p}.mlp.w13", [(f"{l}.mlp.gate", f.ff), (f"{l}.mlp.up", f.ff)]))
            single["mlp.down"] = "mlp.w2"
        out.update({f"{l}.{theirs}": Place(f"{p}.{ours}") for theirs, ours in single.items()})
    return out


def _moe(experts, top, ff, groups, keep, scale) -> MoeSpec:
    return MoeSpec(experts, top, ReluSquareSpec(ff), routing=Routing(groups, keep, scale))


def _big(i: int) -> LayerSpec:
    if i % 4 == 3:
        mixer = DifferentialSpec(32, 4, 64, 128, 0.125, 0.8, QueryTemperature(0.1, 8192), kv_from=i - 4 if i % 8 == 7 else None)
    else:
        mixer = SsmSpec(64, 64, 128, 4, 4)
    return LayerSpec(mixer, plain_glu(6144) if i == 0 else _moe(128, 8, 1152, 8, 4, 2.5))


PRESETS = {
    # plumbing-sized model: both mixers, every kind of feed-forward, a layer on another's keys and values
    "vozirax-tiny": _config([
        LayerSpec(SsmSpec(4, 32, 32, 2, 4, 2), plain_glu(160)),
        LayerSpec(DifferentialSpec(4, 2, 16, 32, 0.3, 0.5, QueryTemperature(0.2, 64)), _moe(8, 2, 64, 4, 2, 1.25)),
        LayerSpec(SsmSpec(6, 16, 48, 1, 3, 1), None),
        LayerSpec(DifferentialSpec(2, 2, 16, 32, 0.25, 0.7, None, kv_from=1), _moe(6, 3, 32, 1, 1, 1.0))], "vozirax-tiny", 512, 128, logit_scale=0.5),
    # layer sizes of a 30B mixture of experts with 3B active parameters: three state-space layers per attention layer
    "vozirax-30B-A3B-shape": _config([_big(i) for i in range(48)], "vozirax-30B-A3B-shape", 151936, 2048),
}
