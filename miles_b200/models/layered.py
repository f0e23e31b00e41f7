"""Decoders described layer by layer: every layer names its own mixer, the mixer's sizes and its feed-forward.

`FamilyConfig` (families.py) gives one set of sizes to a whole model; designs whose layers differ in head counts, windows,
latent ranks or state sizes are a `LayeredConfig`: a tuple of `LayerSpec`s over the building blocks here.

    LatentMixer        latent attention over a paged cache of latents: sliding window, per-head softmax sink, interleaved
                       rotary with optional YaRN frequencies, layers that read another layer's latents (`kv_from`)
    LinearStateMixer   linear attention with a constant decay per head: fp32 state per sequence, gated norm over all heads
    ClampedGLU         gate and up projections with clamped pre-activations
    LayeredModel       hashed-bigram embedding, norms on the sublayers' OUTPUTS with a layer scale, fp32 residual stream

The blocks run in the engine only (paged latents, state slots; no autograd).  What the design keeps in 32 bits — rotary
angles, scores and softmax, norms, the residual sum, recurrent state and decays — is 32-bit in the kernels; matrix products
and activations use the model's dtype (bfloat16, or float32 throughout).

A forward pass takes a ragged batch: any number of new tokens per sequence (`ForwardMeta.ragged`), with sequences that bring
at most `SHORT_Q` tokens last.  Long pieces expand the latents of their window to per-head keys and values; short ones (decode
steps among them) attend to the latents directly with the key up-projection absorbed into the query.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch
import torch.nn as nn

from .. import ops
from ..ops import mixers as MX
from .families import FamilyConfig
from .qwen3 import ForwardMeta, Qwen3Model, _Init


@dataclass(frozen=True)
class YarnScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotary:
    """Rotary embedding of `dims` dimensions in interleaved pairs (2i, 2i + 1)."""

    base: float
    dims: int
    scaling: YarnScaling | None = None

    def table(self) -> tuple[list[float], float]:
        """(angular frequency of every pair, factor on cosine and sine)."""
        half = self.dims // 2
        freq = [self.base ** (-2.0 * i / self.dims) for i in range(half)]
        s = self.scaling
        if s is None:
            return freq, 1.0

        def pair_of(turns: float) -> float:        # the (real-valued) dimension that turns this often over the original context
            return self.dims * math.log(s.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))

        lo = max(math.floor(pair_of(s.fast)), 0)
        hi = min(math.ceil(pair_of(s.slow)), self.dims - 1)
        span = max(hi - lo, 0.001)
        ramp = [min(max((i - lo) / span, 0.0), 1.0) for i in range(half)]
        return [f / s.factor * r + f * (1.0 - r) for f, r in zip(freq, ramp)], 0.1 * math.log(s.factor) + 1.0


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int                       # query / key dimensions without rotation
    rot_dim: int                   # rotated query dimensions per head; the rotated key part is shared by the heads
    vdim: int
    kv_rank: int
    scale: float
    rotary: Rotary
    window: int = 0                # keys a query sees, itself included; 0: all earlier ones
    sink: bool = True              # a learned extra term in every head's softmax denominator
    kv_from: int | None = None     # layer whose cached latents this layer reads instead of writing its own


@dataclass(frozen=True)
class LinearStateSpec:
    heads: int
    dim: int
    vdim: int
    decay: tuple


@dataclass(frozen=True)
class GluSpec:
    ff: int
    limit: float
    alpha: float = 1.702


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentSpec | LinearStateSpec
    mlp: GluSpec | None


@dataclass(frozen=True)
class BigramSpec:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class LayeredConfig(FamilyConfig):
    layer_specs: tuple = ()
    bigram: BigramSpec | None = None

    def with_(self, **kw) -> "LayeredConfig":
        if "num_layers" in kw:                     # fewer layers: the first ones
            kw.setdefault("layer_specs", self.layer_specs[: kw["num_layers"]])
        return super().with_(**kw)

    def num_params(self, active_only: bool = False) -> int:
        n = 2 * self.vocab_size * self.hidden_size + self.hidden_size
        if self.bigram is not None and not active_only:
            n += (self.bigram.buckets + 1) * self.hidden_size
        for s in self.layer_specs:
            n += sum(math.prod(shape) for shape in mixer_shapes(s.mixer, self.hidden_size).values()) + 2 * self.hidden_size
            if s.mlp is not None:
                n += 3 * s.mlp.ff * self.hidden_size + 2 * self.hidden_size
        return n

    def flops_per_token(self, seq_len: int, backward: bool = True) -> float:
        f = 2.0 * (self.num_params(active_only=True) - self.vocab_size * self.hidden_size)
        for s in self.layer_specs:
            m = s.mixer
            if isinstance(m, LatentSpec):
                f += 2.0 * m.heads * (m.dim + m.rot_dim + m.vdim) * min(m.window or seq_len, seq_len / 2.0)
            else:
                f += 4.0 * m.heads * m.dim * m.vdim
        return f * (3.0 if backward else 1.0)

    def to_hf_config(self) -> dict:
        from .nopelorn import to_config

        return to_config(self)


def mixer_shapes(m, hidden: int) -> dict[str, tuple]:
    """Parameter shapes of a mixer (projections of one input stacked so that each input is multiplied once)."""
    if isinstance(m, LatentSpec):
        rows = m.heads * (m.dim + m.rot_dim) + (0 if m.kv_from is not None else m.kv_rank + m.rot_dim)
        out = {"w_in": (rows, hidden), "w_ukv": (m.heads * (m.dim + m.vdim), m.kv_rank), "wo": (hidden, m.heads * m.vdim)}
        if m.kv_from is None:
            out["kv_norm"] = (m.kv_rank,)
        if m.sink:
            out["sink"] = (m.heads,)
        return out
    return {"w_in": (m.heads * 2 * (m.dim + m.vdim), hidden), "norm": (m.heads * m.vdim,), "wo": (hidden, m.heads * m.vdim)}


class _Mixer(nn.Module):
    def __init__(self, spec, hidden: int, std: float, dtype, device, gen, tag: str):
        super().__init__()
        self.spec = spec
        for name, shape in mixer_shapes(spec, hidden).items():
            if len(shape) == 2:
                t = gen(f"{tag}.{name}", shape, std, dtype, device)
            else:
                t = (torch.zeros if name == "sink" else torch.ones)(shape, dtype=dtype, device=device)
            setattr(self, name, nn.Parameter(t))


class LatentMixer(_Mixer):
    def __init__(self, spec: LatentSpec, *a):
        super().__init__(spec, *a)
        freq, self.magnitude = spec.rotary.table()
        self.register_buffer("freq", torch.tensor(freq, dtype=torch.float64, device=self.wo.device), persistent=False)
        self.layout = MX.LatentLayout(spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank)

    def forward(self, proj, meta: ForwardMeta, layer: int, eps: float):
        s = self.spec
        cache = meta.kv_cache[layer if s.kv_from is None else s.kv_from][0]
        return MX.latent_attention(proj, self.layout, cache, meta, freq=self.freq, magnitude=self.magnitude, scale=s.scale,
                                   window=s.window, sink=getattr(self, "sink", None), w_ukv=self.w_ukv,
                                   kv_norm=getattr(self, "kv_norm", None), eps=eps)


class LinearStateMixer(_Mixer):
    def __init__(self, spec: LinearStateSpec, *a):
        super().__init__(spec, *a)
        assert len(spec.decay) == spec.heads, "one decay per head"
        self.register_buffer("decay", torch.tensor(spec.decay, dtype=torch.float64, device=self.wo.device).float(), persistent=False)

    def forward(self, proj, meta: ForwardMeta, layer: int, eps: float):
        s = self.spec
        return MX.linear_state_attention(proj, s.heads, s.dim, s.vdim, self.decay, meta.states[layer], meta, self.norm, eps)


class ClampedGLU(nn.Module):
    def __init__(self, spec: GluSpec, hidden: int, std: float, dtype, device, gen, tag: str):
        super().__init__()
        self.spec = spec
        self.w13 = nn.Parameter(gen(f"{tag}.w13", (2 * spec.ff, hidden), std, dtype, device))
        self.w2 = nn.Parameter(gen(f"{tag}.w2", (hidden, spec.ff), std, dtype, device))

    def forward(self, proj):
        return ops.linear(MX.clamped_glu(proj, self.spec.limit, self.spec.alpha), self.w2)


class _Stream:
    """The fp32 residual and a sublayer output that has not been added to it yet.

    `project` adds the pending output (norm, layer scale, residual sum) and multiplies the new residual by a weight: one kernel
    for a handful of rows, a norm kernel and a GEMM otherwise."""

    def __init__(self, x, xb, eps: float):
        self.x, self.xb, self.eps, self.pending = x, xb, eps, None

    def project(self, w):
        if self.pending is None:
            return ops.linear(self.xb, w)
        y, nw, ls = self.pending
        self.pending = None
        if MX.few_row_projection(y, w):
            out, self.x = MX.output_norm_linear(self.x, y, nw, ls, self.eps, w)
            self.xb = None
            return out
        self.x, self.xb = MX.output_norm_residual(self.x, y, nw, ls, self.eps)
        return ops.linear(self.xb, w)

    def add(self, y, nw, ls):
        self.pending = (y, nw, ls)

    def finish(self, final_w):
        y, nw, ls = self.pending
        return MX.output_norm_residual(self.x, y, nw, ls, self.eps, final_w=final_w)[1]

    def value(self):
        """The residual with everything added (debugging and tests)."""
        if self.pending is None:
            return self.x.clone()
        y, nw, ls = self.pending
        return MX.output_norm_residual(self.x.clone(), y, nw, ls, self.eps)[0]


class LayeredLayer(nn.Module):
    def __init__(self, spec: LayerSpec, cfg: LayeredConfig, dtype, device, gen, layer: int):
        super().__init__()
        self.layer, self.eps = layer, cfg.rms_eps
        H, std = cfg.hidden_size, cfg.init_std

        def vec():
            return nn.Parameter(torch.ones(H, dtype=dtype, device=device))

        kind = LatentMixer if isinstance(spec.mixer, LatentSpec) else LinearStateMixer
        self.norm1, self.ls1 = vec(), vec()
        self.mix = kind(spec.mixer, H, std, dtype, device, gen, f"L{layer}.mix")
        self.mlp = None
        if spec.mlp is not None:
            self.norm2, self.ls2 = vec(), vec()
            self.mlp = ClampedGLU(spec.mlp, H, std, dtype, device, gen, f"L{layer}.mlp")

    def forward(self, st: _Stream, meta: ForwardMeta):
        o = self.mix(st.project(self.mix.w_in), meta, self.layer, self.eps)
        st.add(ops.linear(o, self.mix.wo), self.norm1, self.ls1)
        if self.mlp is not None:
            st.add(self.mlp(st.project(self.mlp.w13)), self.norm2, self.ls2)


class LayeredModel(Qwen3Model):
    """Decoder assembled from `LayeredConfig.layer_specs`; the engine's interface of `Qwen3Model`."""

    ragged_batches = True          # the engine hands this model `ForwardMeta.ragged` batches (any mix of pieces and decode steps)
    supports_kv_cache = True

    def __init__(self, cfg: LayeredConfig, ps=None, dtype=torch.bfloat16, device="cpu", seed: int = 0):
        super().__init__(cfg.with_(num_layers=0), ps, dtype=dtype, device=device, seed=seed, layer_range=(0, 0))
        assert self.ps.tp_size == 1 and self.ps.pp_size == 1 and self.ps.cp_size == 1, "layered models run on one rank"
        assert len(cfg.layer_specs) == cfg.num_layers, f"{cfg.num_layers} layers, {len(cfg.layer_specs)} described"
        self.cfg = cfg
        gen = _Init(seed)
        self.layer_range = (0, cfg.num_layers)
        self.has_embed = self.has_head = True
        for i, s in enumerate(cfg.layer_specs):
            m = s.mixer
            if isinstance(m, LatentSpec) and m.kv_from is not None:
                src = cfg.layer_specs[m.kv_from].mixer
                assert m.kv_from < i and isinstance(src, LatentSpec) and src.kv_from is None and (src.kv_rank, src.rot_dim) == (
                    m.kv_rank, m.rot_dim), f"layer {i} cannot read the latents of layer {m.kv_from}"
        self.layers = nn.ModuleList(LayeredLayer(s, cfg, dtype, device, gen, l) for l, s in enumerate(cfg.layer_specs))
        self.bigram = None
        if cfg.bigram is not None:
            self.bigram = nn.Parameter(gen("bigram", (cfg.bigram.buckets + 1, cfg.hidden_size), cfg.init_std, dtype, device))
        self.num_moe_layers = 0

    # ---- what the engine keeps per token and per sequence ------------------------------------------------------------
    def kv_rows(self) -> dict[int, tuple]:
        """Cache row shapes per token of every layer that writes one."""
        return {l.layer: ((l.mix.layout.pitch,),) for l in self.layers if isinstance(l.mix, LatentMixer) and l.mix.spec.kv_from is None}

    def state_shapes(self) -> dict[int, tuple]:
        """fp32 state per sequence of every recurrent layer."""
        return {l.layer: (l.mix.spec.heads, l.mix.spec.dim, l.mix.spec.vdim) for l in self.layers if isinstance(l.mix, LinearStateMixer)}

    def forward(self, tokens, meta: ForwardMeta, hidden_in=None, inputs_embeds=None):
        if torch.is_grad_enabled():
            raise NotImplementedError("layered models run in the engine only: no backward pass is built for their mixers")
        assert meta.ragged is not None, "layered models take ragged engine batches"
        big = self.cfg.bigram
        x, xb = MX.bigram_embedding(tokens, meta.prev_tokens, self.embed, self.bigram,
                                    (big.buckets, big.mul_prev, big.mul_cur) if big is not None else None)
        st = _Stream(x, xb, self.cfg.rms_eps)
        for layer in self.layers:
            layer(st, meta)
            if meta.record_residual is not None:
                meta.record_residual.append(st.value())
        return st.finish(self.norm)
