"""Ronupel: `config.json` ⇄ `LayeredConfig`, checkpoint names → this package's parameters.

A Ronupel model lists its layers one by one; in each, grouped-query attention (sliding window that keeps the first tokens, softmax
sink, norm over the whole query and key projection, linearly scaled rotary) and a mixture of clamped experts with a shared one read
the same normed residual.  A range of layers may run several times with the same weights.  The head is the embedding table.
Checkpoint tensors are called `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`, `embed`, `final.norm`; here what reads one input is stacked
along the rows (`w_in`), what adds to one sum along the columns (`w_out`), and a layer's experts form one tensor.
"""
from __future__ import annotations

from .layered import AttentionSpec, GluSpec, LayeredConfig, LayerSpec, LinearScaling, LoopSpec, MoeSpec, Rotary

ARCHITECTURE = "Ronupel"


def _mixer(kind: str, m: dict) -> AttentionSpec:
    if kind != "attention":
        raise ValueError(f"unknown Ronupel mixer '{kind}'")
    r, mask = m.get("rot"), m.get("mask") or {}
    sc = (r or {}).get("scaling")
    return AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"],
                         rotary=Rotary(r["base"], r["dims"], LinearScaling(sc["factor"]) if sc else None) if r else None,
                         window=mask.get("size") or 0, keep_first=(mask.get("keep_first") or 0) if mask.get("size") else 0)


def _mlp(m: dict | None) -> MoeSpec | None:
    if m is None:
        return None
    if m["kind"] != "moe":
        raise ValueError(f"unknown Ronupel feed-forward '{m['kind']}'")
    e, s = m["expert"], m.get("shared")
    return MoeSpec(experts=m["router"]["experts"], top=m["router"]["top"], expert=GluSpec(e["ff"], e["limit"]),
                   shared=GluSpec(s["ff"], s["limit"]) if s else None)


def from_config(cfg: dict) -> LayeredConfig:
    layers = tuple(LayerSpec(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in cfg["layers"])
    loop = cfg.get("loop")
    moes = [l.mlp for l in layers if l.mlp is not None]
    return LayeredConfig(name=cfg.get("name", "ronupel"), family="ronupel", vocab_size=cfg["vocab"], hidden_size=cfg["width"],
                         num_layers=len(layers), num_heads=1, num_kv_heads=1, head_dim=0, ffn_hidden_size=0,
                         rms_eps=cfg["norm"]["eps"], tie_embeddings=True, layer_specs=layers, block="parallel",
                         loop=LoopSpec(loop["start"], loop["stop"], loop["times"]) if loop else None,
                         # what the engine records of the routing: the widest layer's choices
                         num_experts=max((m.experts for m in moes), default=0), moe_topk=max((m.top for m in moes), default=0))


def to_config(cfg: LayeredConfig) -> dict:
    def layer(s: LayerSpec) -> dict:
        m, f = s.mixer, s.mlp
        d = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
        if m.rotary is not None:
            d["rot"] = {"base": m.rotary.base, "dims": m.rotary.dims}
            if m.rotary.scaling is not None:
                d["rot"]["scaling"] = {"factor": m.rotary.scaling.factor}
        if m.window:
            d["mask"] = {"size": m.window, "keep_first": m.keep_first}
        mlp = None
        if f is not None:
            mlp = {"kind": "moe", "router": {"experts": f.experts, "top": f.top}, "expert": {"ff": f.expert.ff, "limit": f.expert.limit}}
            if f.shared is not None:
                mlp["shared"] = {"ff": f.shared.ff, "limit": f.shared.limit}
        return {"type": "attention", "mixer": d, "mlp": mlp}

    out = {"architecture": ARCHITECTURE, "name": cfg.name, "vocab": cfg.vocab_size, "width": cfg.hidden_size,
           "norm": {"eps": cfg.rms_eps}, "layers": [layer(s) for s in cfg.layer_specs]}
    if cfg.loop is not None:
        out["loop"] = {"start": cfg.loop.start, "stop": cfg.loop.stop, "times": cfg.loop.times}
    return out


def tensors(cfg: LayeredConfig) -> dict:
    from .designs import Place, rows_of

    H = cfg.hidden_size
    out = {"embed": Place("embed"), "final.norm": Place("norm")}
    for i, s in enumerate(cfg.layer_specs):
        m, f, l, p = s.mixer, s.mlp, f"l{i}", f"layers.{i}"
        heads, dense = m.heads * m.vdim, s.dense
        rows = [(f"{l}.mix.q", m.heads * m.dim), (f"{l}.mix.k", m.kv_heads * m.dim), (f"{l}.mix.v", m.kv_heads * m.vdim)]
        out[f"{l}.mix.o"] = Place(f"{p}.w_out", ((0, H), (0, heads)))
        if dense is not None:
            rows += [(f"{l}.mlp.shared.gate", dense.ff), (f"{l}.mlp.shared.up", dense.ff)]
            out[f"{l}.mlp.shared.down"] = Place(f"{p}.w_out", ((0, H), (heads, heads + dense.ff)))
        out.update(rows_of(f"{p}.w_in", rows))
        single = {"norm1": "norm1", "mix.q.norm": "mix.q_norm", "mix.k.norm": "mix.k_norm", "mix.sink": "mix.sink"}
        if f is not None:
            single.update({"mlp.router": "mlp.router", "mlp.router.b": "mlp.bias"})
            F = f.expert.ff
            for e in range(f.experts):
                out[f"{l}.mlp.e{e}.gate"] = Place(f"{p}.mlp.w13", ((e, e + 1), (0, F)), True)
                out[f"{l}.mlp.e{e}.up"] = Place(f"{p}.mlp.w13", ((e, e + 1), (F, 2 * F)), True)
                out[f"{l}.mlp.e{e}.down"] = Place(f"{p}.mlp.w2", ((e, e + 1),), True)
        out.update({f"{l}.{theirs}": Place(f"{p}.{ours}") for theirs, ours in single.items()})
    return out


def _layer(heads, kv_heads, dim, vdim, window, keep, experts, top, ff, shared, limit=7.0, scaling=1.0, base=1e6, rot=None) -> LayerSpec:
    return LayerSpec(AttentionSpec(heads, kv_heads, dim, vdim, dim ** -0.5, Rotary(base, rot or dim, LinearScaling(scaling)), window, keep),
                     MoeSpec(experts, top, GluSpec(ff, limit), GluSpec(shared, limit)))


def _preset(name, vocab, width, layers, loop) -> LayeredConfig:
    moes = [l.mlp for l in layers if l.mlp is not None]
    return LayeredConfig(name=name, family="ronupel", vocab_size=vocab, hidden_size=width, num_layers=len(layers), num_heads=1, num_kv_heads=1,
                         head_dim=0, ffn_hidden_size=0, tie_embeddings=True, layer_specs=tuple(layers), block="parallel", loop=loop,
                         num_experts=max(m.experts for m in moes), moe_topk=max(m.top for m in moes))


PRESETS = {
    # plumbing-sized model: layers of unlike sizes, one without a feed-forward, two passes over the middle
    "ronupel-tiny": _preset("ronupel-tiny", 512, 128, [
        _layer(4, 2, 32, 32, 48, 8, 6, 2, 64, 96, scaling=2.0, rot=16), _layer(6, 2, 16, 32, 24, 4, 8, 3, 32, 64),
        LayerSpec(AttentionSpec(4, 1, 32, 16, 0.2, Rotary(2e4, 32, LinearScaling(4.0)), 32, 5), None),
        _layer(2, 2, 64, 64, 40, 0, 4, 1, 96, 32)], LoopSpec(1, 3, 2)),
    # layer sizes of a 30B mixture of experts with 3B active parameters; 44 layers, 48 layer runs
    "ronupel-30B-A3B-shape": _preset("ronupel-30B-A3B-shape", 151936, 2048,
                                     [_layer(32, 4, 128, 128, 1024, 64, 128, 8, 768, 768, scaling=4.0) for _ in range(44)], LoopSpec(4, 8, 2)),
}
