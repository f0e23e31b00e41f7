"""Senadra: `config.json` ⇄ `LayeredConfig`, checkpoint names → this package's parameters.

A Senadra model lists its layers one by one: a gated delta rule with a decay per key channel, latent attention with latent queries, or
grouped-query attention inside chunks with a distance bias (which may read an earlier layer's keys and values); then a feed-forward or
none; then a token input of its own.  Every sublayer sits behind a norm, its output counts `residual_mult` times, and the logits pass a
soft cap.  Checkpoint tensors are called `l<i>.norm1/2`, `l<i>.mix.*`, `l<i>.mlp.*`, `l<i>.side.*`, `embed`, `side.embed`, `final.norm`,
`head`; here the projections of one input are stacked along the rows (`mix.w_in`, `mix.w_ukv`), as are a layer's convolutions.

The inner sizes of the delta rule's two-step projections (decays, output gate) are those of the tensors; a configuration without
a checkpoint names them (`decay_rank`, `gate_rank`).
"""
from __future__ import annotations

from .layered import AttentionSpec, DeltaSpec, LatentSpec, LayeredConfig, LayerSpec, Rotary, XieluSpec

ARCHITECTURE = "Senadra"
SIZES_FROM_TENSORS = True


def _mixer(kind: str, m: dict, shapes: dict, prefix: str):
    if kind == "channel_delta":
        def rank(key, tensor):
            if key in m:
                return m[key]
            if prefix + tensor not in shapes:
                raise ValueError(f"the configuration gives no '{key}' and there is no tensor {prefix + tensor} to take it from")
            return shapes[prefix + tensor][0]

        return DeltaSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], conv=m["conv"],
                         decay_rank=rank("decay_rank", "a1"), gate_rank=rank("gate_rank", "g1"))
    if kind == "latent_attention":
        r = m["rot"]
        assert r["dims"] == m["rot_dim"], "the rotation covers the rotated part of each head"
        return LatentSpec(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"], scale=m["scale"],
                          rotary=Rotary(r["base"], r["dims"]), sink=False, q_rank=m["q_rank"], gate=True)
    if kind == "attention":
        return AttentionSpec(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], qk_norm=False, sink=False,
                             chunk=(m.get("mask") or {}).get("size") or 0, distance_bias=True, value_norm=True, gate=True,
                             kv_from=m.get("kv_from"))
    raise ValueError(f"unknown Senadra mixer '{kind}'")


def _mlp(m: dict | None):
    if m is None:
        return None
    if m["kind"] != "dense":
        raise ValueError(f"unknown Senadra feed-forward '{m['kind']}'")
    return XieluSpec(m["ff"])


def _config(layers, name: str, vocab: int, width: int, eps: float = 1e-6, mult: float = 1.0, softcap: float = 0.0, side: int = 0) -> LayeredConfig:
    return LayeredConfig(name=name, family="senadra", vocab_size=vocab, hidden_size=width, num_layers=len(layers), num_heads=1, num_kv_heads=1,
                         head_dim=0, ffn_hidden_size=0, rms_eps=eps, layer_specs=tuple(layers), block="pre_norm", residual_mult=mult,
                         logit_softcap=softcap, token_side=side)


def from_config(cfg: dict, shapes: dict | None = None) -> LayeredConfig:
    layers = [LayerSpec(_mixer(l["type"], l["mixer"], shapes or {}, f"l{i}.mix."), _mlp(l.get("mlp"))) for i, l in enumerate(cfg["layers"])]
    return _config(layers, cfg.get("name", "senadra"), cfg["vocab"], cfg["width"], cfg["norm"]["eps"], cfg["residual_mult"],
                   cfg.get("logit_softcap") or 0.0, (cfg.get("token_side") or {}).get("dim") or 0)


def to_config(cfg: LayeredConfig) -> dict:
    def layer(s: LayerSpec) -> dict:
        m = s.mixer
        if isinstance(m, DeltaSpec):
            kind, d = "channel_delta", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.conv,
                                        "decay_rank": m.decay_rank, "gate_rank": m.gate_rank}
        elif isinstance(m, LatentSpec):
            kind, d = "latent_attention", {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                                           "q_rank": m.q_rank, "scale": m.scale, "rot": {"base": m.rotary.base, "dims": m.rotary.dims}}
        else:
            kind, d = "attention", {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
            if m.chunk:
                d["mask"] = {"size": m.chunk}
            if m.kv_from is not None:
                d["kv_from"] = m.kv_from
        return {"type": kind, "mixer": d, "mlp": None if s.mlp is None else {"kind": "dense", "ff": s.mlp.ff}}

    out = {"architecture": ARCHITECTURE, "name": cfg.name, "vocab": cfg.vocab_size, "width": cfg.hidden_size, "norm": {"eps": cfg.rms_eps},
           "residual_mult": cfg.residual_mult, "layers": [layer(s) for s in cfg.layer_specs]}
    if cfg.logit_softcap:
        out["logit_softcap"] = cfg.logit_softcap
    if cfg.token_side:
        out["token_side"] = {"dim": cfg.token_side}
    return out


def tensors(cfg: LayeredConfig) -> dict:
    from .designs import Place, rows_of

    out = {"embed": Place("embed"), "final.norm": Place("norm"), "head": Place("lm_head")}
    if cfg.token_side:
        out["side.embed"] = Place("side_embed")
    for i, s in enumerate(cfg.layer_specs):
        m, l, p = s.mixer, f"l{i}", f"layers.{i}"
        single = {"norm1": "norm1", "mix.o": "mix.wo"}
        if isinstance(m, DeltaSpec):
            k, v = m.kv_heads * m.dim, m.heads * m.vdim
            out.update(rows_of(f"{p}.mix.w_in", [(f"{l}.mix.q", k), (f"{l}.mix.k", k), (f"{l}.mix.v", v), (f"{l}.mix.a1", m.decay_rank),
                                                 (f"{l}.mix.g1", m.gate_rank), (f"{l}.mix.b", m.heads)]))
            out.update(rows_of(f"{p}.mix.conv", [(f"{l}.mix.q.conv", k), (f"{l}.mix.k.conv", k), (f"{l}.mix.v.conv", v)]))
            single.update({"mix.a2": "mix.w_a", "mix.g2": "mix.w_g", "mix.A_log": "mix.A_log", "mix.dt_bias": "mix.dt_bias", "mix.norm": "mix.norm"})
        elif isinstance(m, LatentSpec):
            rows = [(f"{l}.mix.dq", m.q_rank), (f"{l}.mix.dkv", m.kv_rank + m.rot_dim), (f"{l}.mix.g", m.heads * m.vdim)]
            out.update(rows_of(f"{p}.mix.w_in", rows))
            out.update(rows_of(f"{p}.mix.w_ukv", [(f"{l}.mix.uk", m.heads * m.dim), (f"{l}.mix.uv", m.heads * m.vdim)]))
            single.update({"mix.dq.norm": "mix.q_norm", "mix.uq": "mix.w_uq", "mix.dkv.norm": "mix.kv_norm"})
        else:
            rows = [(f"{l}.mix.q", m.heads * m.dim)]
            if m.kv_from is None:
                rows += [(f"{l}.mix.k", m.kv_heads * m.dim), (f"{l}.mix.v", m.kv_heads * m.vdim)]
            out.update(rows_of(f"{p}.mix.w_in", rows + [(f"{l}.mix.g", m.heads * m.vdim)]))
            single.update({"mix.r1": "mix.r1", "mix.r2": "mix.r2"})
        if s.mlp is not None:
            single.update({"norm2": "norm2", "mlp.up": "mlp.w13", "mlp.down": "mlp.w2", "mlp.act": "mlp.act"})
        if cfg.token_side:
            single.update({f"side.{n}": f"side.{n}" for n in ("gate", "proj", "norm")})
        out.update({f"{l}.{theirs}": Place(f"{p}.{ours}") for theirs, ours in single.items()})
    return out


def _big(i: int) -> LayerSpec:
    if i % 4 == 3:
        mixer = LatentSpec(32, 128, 64, 128, 512, 0.0722, Rotary(1e6, 64), sink=False, q_rank=1536, gate=True)
    elif i % 4 == 1:
        mixer = AttentionSpec(32, 8, 128, 128, 0.0884, qk_norm=False, sink=False, chunk=2048, distance_bias=True, value_norm=True, gate=True,
                              kv_from=i - 4 if i % 8 == 5 else None)
    else:
        mixer = DeltaSpec(32, 32, 128, 128, 4, 128, 128)
    return LayerSpec(mixer, XieluSpec(9728))


def _chunked(heads, kv_heads, dim, vdim, scale, chunk, kv_from=None) -> AttentionSpec:
    return AttentionSpec(heads, kv_heads, dim, vdim, scale, qk_norm=False, sink=False, chunk=chunk, distance_bias=True, value_norm=True, gate=True,
                         kv_from=kv_from)


PRESETS = {
    # plumbing-sized model: every mixer, a layer without feed-forward, a layer on another's keys and values
    "senadra-tiny": _config([
        LayerSpec(DeltaSpec(4, 2, 16, 32, 4, 16, 24), XieluSpec(160)),
        LayerSpec(_chunked(4, 2, 16, 32, 0.3, 40), XieluSpec(160)),
        LayerSpec(LatentSpec(4, 32, 16, 32, 48, 0.15, Rotary(20000.0, 16), sink=False, q_rank=64, gate=True), None),
        LayerSpec(_chunked(8, 2, 16, 32, 0.25, 64, kv_from=1), XieluSpec(96)),
        LayerSpec(DeltaSpec(3, 3, 24, 16, 3, 8, 8), XieluSpec(96))], "senadra-tiny", 512, 128, mult=0.5, softcap=20.0, side=16),
    # layer sizes of a mid-sized model: two delta-rule layers, one chunked and one latent attention layer per group of four
    "senadra-4B-shape": _config([_big(i) for i in range(36)], "senadra-4B-shape", 151936, 2560, mult=0.4, softcap=30.0, side=256),
}
