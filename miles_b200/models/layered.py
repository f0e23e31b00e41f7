"""Decoders described layer by layer: every layer names its own mixer, the mixer's sizes and its feed-forward.

`FamilyConfig` (families.py) gives one set of sizes to a whole model; designs whose layers differ in head counts, windows,
latent ranks or state sizes are a `LayeredConfig`: a tuple of `LayerSpec`s over the building blocks here.

    LatentMixer        latent attention over a paged cache of latents: sliding window, per-head softmax sink, interleaved
                       rotary with optional YaRN frequencies, layers that read another layer's latents (`kv_from`)
                       queries through a latent of their own, output gate
    LinearStateMixer   linear attention with a constant decay per head: fp32 state per sequence, gated norm over all heads
    DeltaMixer         gated delta rule with a decay per key channel: short convolutions, unit queries and keys, fp32 state, gated norm
                       per head
    AttentionMixer     grouped-query attention over a paged cache of keys and values: sliding window that keeps the first tokens, or
                       chunks; per-head softmax sink or distance bias, RMS norm over a token's whole query (key) projection or
                       over its values, interleaved rotary, output gate; may read another layer's keys and values
    DifferentialMixer  two softmax maps per head over the same values, the second subtracted with a learned weight; norms per head and
                       map, a query temperature that grows with the position, a gate per head; may read another layer's keys and values
    SsmMixer           state-space layer with a scalar decay per head and token: short convolution, fp32 state, gate, norm in parts
    ClampedGLU         gate and up projections with clamped pre-activations (a limit of infinity: plain silu(gate) · up)
    Xielu              ungated feed-forward with a learned quadratic / exponential activation
    TokenSide          per-layer token input: a second look-up per token and layer, gated by the residual, normed and added
    RoutedExperts      clamped gated experts or ungated ones with a squared relu; chosen by the `top` largest of biased fp32 logits
                       with weights by their softmax, or by corrected sigmoid scores among the best groups (`Routing`)
    LayeredModel       hashed-bigram embedding and / or sinusoidal positions, fp32 residual stream, layers in one of four arrangements
                       (`LayeredConfig.block`):
                       "output_norm"  mixer, then feed-forward, norms on the sublayers' OUTPUTS with a layer scale
                       "parallel"     one norm in front; mixer and feed-forward read it side by side and are added together
                       "two_norms"    mixer and feed-forward side by side, each behind a norm and before a layer scale of its own
                       "pre_norm"     mixer, then feed-forward, then token input, each behind a norm in front and times one factor
                       A range of layers may run several times with the same weights (`LoopSpec`), each pass on its own cache.

The blocks run in the engine only (paged latents, state slots; no autograd).  What the design keeps in 32 bits — rotary
angles, scores and softmax, norms, the residual sum, recurrent state and decays — is 32-bit in the kernels; matrix products
and activations use the model's dtype (bfloat16, or float32 throughout).

A forward pass takes a ragged batch: any number of new tokens per sequence (`ForwardMeta.ragged`), with sequences that bring
at most `SHORT_Q` tokens last.  Latent attention expands the latents of a long piece's window to per-head keys and values; short pieces (decode steps
among them) attend to the latents directly with the key up-projection absorbed into the query.  Grouped-query attention runs long
pieces as query tiles over the cached pages and short ones token by token.
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
class LinearScaling:
    """Positions count `factor` times slower."""

    factor: float


@dataclass(frozen=True)
class Rotary:
    """Rotary embedding of `dims` dimensions in interleaved pairs (2i, 2i + 1)."""

    base: float
    dims: int
    scaling: YarnScaling | LinearScaling | None = None

    def table(self) -> tuple[list[float], float]:
        """(angular frequency of every pair, factor on cosine and sine)."""
        half = self.dims // 2
        freq = [self.base ** (-2.0 * i / self.dims) for i in range(half)]
        s = self.scaling
        if s is None:
            return freq, 1.0
        if isinstance(s, LinearScaling):
            return [f / s.factor for f in freq], 1.0

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
    q_rank: int = 0                # queries come from a normed latent of this size (0: straight from the input)
    gate: bool = False             # outputs times the sigmoid of a projection of the input


@dataclass(frozen=True)
class DeltaSpec:
    """Gated delta rule: per head S ← diag(g)·S, S ← S + β k (v − Sᵀk)ᵀ, o = Sᵀq, with a decay g per key channel."""

    heads: int
    kv_heads: int                  # query / key heads; heads share them in equal groups
    dim: int
    vdim: int
    conv: int                      # columns of the causal convolutions
    decay_rank: int                # inner size of the decays' two projections
    gate_rank: int                 # … of the output gate's


@dataclass(frozen=True)
class LinearStateSpec:
    heads: int
    dim: int
    vdim: int
    decay: tuple


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int                       # query / key size per head
    vdim: int
    scale: float
    rotary: Rotary | None = None   # rotates the first `rotary.dims` dimensions of queries and keys
    window: int = 0                # keys a query sees, itself included; 0: all earlier ones
    keep_first: int = 0            # tokens at the start of a sequence that stay visible whatever the window
    qk_norm: bool = True           # RMS norm over a token's whole query (key) projection, before the heads are rotated
    sink: bool = True              # a learned extra term in every head's softmax denominator
    chunk: int = 0                 # tokens see their own chunk of this many positions only (0: no chunks)
    distance_bias: bool = False    # r1 · ln(1 + r2 · distance) per head off the scores
    value_norm: bool = False       # every head's values over their root mean square
    gate: bool = False             # outputs times the sigmoid of a projection of the input
    kv_from: int | None = None     # layer whose cached keys and values this layer reads instead of writing its own


@dataclass(frozen=True)
class QueryTemperature:
    """Queries at position p count 1 + coef · ln(⌊(p + 1) / every⌋ + 1) times."""

    coef: float
    every: float


@dataclass(frozen=True)
class DifferentialSpec:
    heads: int
    kv_heads: int
    dim: int                       # query / key size of one of a head's two maps
    vdim: int
    scale: float
    diff: float                    # what the weight of the second map starts from; outputs count 1 − diff times
    temperature: QueryTemperature | None = None
    kv_from: int | None = None     # layer whose cached keys and values this layer reads instead of writing its own


@dataclass(frozen=True)
class SsmSpec:
    heads: int
    vdim: int
    state: int
    groups: int                    # heads of a group share B and C
    conv: int                      # columns of the causal convolution
    norm_groups: int = 1           # parts of the output that are normed by themselves


@dataclass(frozen=True)
class GluSpec:
    ff: int
    limit: float = math.inf
    alpha: float = 1.702
    shift: float = 1.0             # added to the up projection


def plain_glu(ff: int) -> GluSpec:
    """silu(gate) · up"""
    return GluSpec(ff, math.inf, 1.0, 0.0)


@dataclass(frozen=True)
class ReluSquareSpec:
    """No gate: down(relu(up)²)."""

    ff: int


@dataclass(frozen=True)
class XieluSpec:
    """No gate: down(xielu(up)), an activation with two learned numbers."""

    ff: int


@dataclass(frozen=True)
class MoeSpec:
    experts: int
    top: int
    expert: GluSpec | ReluSquareSpec
    shared: GluSpec | None = None  # runs for every token and is added
    routing: MX.Routing | None = None    # None: softmax over the chosen logits (with a bias per expert)

    @property
    def up_rows(self) -> int:
        """Rows of an expert's input projection."""
        return self.expert.ff * (2 if isinstance(self.expert, GluSpec) else 1)


@dataclass(frozen=True)
class LayerSpec:
    mixer: LatentSpec | LinearStateSpec | AttentionSpec | DifferentialSpec | SsmSpec | DeltaSpec
    mlp: GluSpec | XieluSpec | MoeSpec | None

    @property
    def dense(self) -> GluSpec | XieluSpec | None:
        """The feed-forward every token passes (all of it, or the shared expert beside routed ones)."""
        return self.mlp.shared if isinstance(self.mlp, MoeSpec) else self.mlp


@dataclass(frozen=True)
class LoopSpec:
    """Layers start … stop − 1 run `times` times in a row; the embedding output is added before each pass but the first."""

    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class BigramSpec:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class LayeredConfig(FamilyConfig):
    layer_specs: tuple = ()
    bigram: BigramSpec | None = None
    block: str = "output_norm"         # or "parallel", "two_norms", "pre_norm"
    loop: LoopSpec | None = None
    norm_shift: float = 0.0            # what norm weights are added to ("two_norms")
    position_base: float = 0.0         # sinusoidal position vectors are added to the embedding (0: none)
    logit_scale: float = 1.0
    logit_softcap: float = 0.0         # logits ← cap · tanh(logits / cap) (0: as they are)
    residual_mult: float = 1.0         # factor on what sublayers add ("pre_norm")
    token_side: int = 0                # size of the per-layer token input (0: none; "pre_norm")

    def with_(self, **kw) -> "LayeredConfig":
        if "num_layers" in kw:                     # fewer layers: the first ones
            n = kw["num_layers"]
            kw.setdefault("layer_specs", self.layer_specs[:n])
            if self.loop is not None and self.loop.stop > n:
                kw.setdefault("loop", LoopSpec(self.loop.start, n, self.loop.times) if self.loop.start < n else None)
        return super().with_(**kw)

    def runs(self) -> list[tuple[int, bool]]:
        """The layer runs of a forward pass in order: (layer, the embedding output is added before it).  Caches and states belong to
        runs: run r of this list owns entry r."""
        if self.loop is None:
            return [(i, False) for i in range(self.num_layers)]
        lo, hi, n = self.loop.start, self.loop.stop, self.loop.times
        return ([(i, False) for i in range(lo)] + [(i, t > 0 and i == lo) for t in range(n) for i in range(lo, hi)]
                + [(i, False) for i in range(hi, self.num_layers)])

    def layer_is_moe(self, layer: int) -> bool:
        return isinstance(self.layer_specs[layer].mlp, MoeSpec)

    @property
    def num_moe_layers(self) -> int:
        return sum(self.layer_is_moe(l) for l, _ in self.runs())

    def num_params(self, active_only: bool = False) -> int:
        """Parameters; `active_only`: those a token meets, each as often as it meets it, without the embedding look-ups."""
        H = self.hidden_size
        n = H + self.vocab_size * H * (1 if self.tie_embeddings else 2)
        if self.bigram is not None and not active_only:
            n += (self.bigram.buckets + 1) * H
        if not active_only:
            n += self.vocab_size * self.num_layers * self.token_side
        for i in [l for l, _ in self.runs()] if active_only else range(self.num_layers):
            s = self.layer_specs[i]
            n += sum(math.prod(shape) for shape in layer_shapes(s, self).values())
            if active_only and isinstance(s.mlp, MoeSpec):
                n -= (s.mlp.experts - s.mlp.top) * (s.mlp.up_rows + s.mlp.expert.ff) * H
        return n

    def flops_per_token(self, seq_len: int, backward: bool = True) -> float:
        f = 2.0 * (self.num_params(active_only=True) - (0 if self.tie_embeddings else self.vocab_size * self.hidden_size))
        for i, _ in self.runs():
            m = self.layer_specs[i].mixer
            if isinstance(m, LatentSpec):
                f += 2.0 * m.heads * (m.dim + m.rot_dim + m.vdim) * min(m.window or seq_len, seq_len / 2.0)
            elif isinstance(m, AttentionSpec):
                f += 2.0 * m.heads * (m.dim + m.vdim) * min(m.window + m.keep_first if m.window else (m.chunk or seq_len) / 2.0, seq_len / 2.0)
            elif isinstance(m, DeltaSpec):
                f += 6.0 * m.heads * m.dim * m.vdim
            elif isinstance(m, DifferentialSpec):
                f += 4.0 * m.heads * (m.dim + m.vdim) * seq_len / 2.0
            elif isinstance(m, SsmSpec):
                f += 4.0 * m.heads * m.state * m.vdim
            else:
                f += 4.0 * m.heads * m.dim * m.vdim
        return f * (3.0 if backward else 1.0)

    def to_hf_config(self) -> dict:
        from .designs import DESIGNS

        return DESIGNS[self.family].to_config(self)


def mixer_shapes(m, hidden: int) -> dict[str, tuple]:
    """Parameter shapes of a mixer (projections of one input stacked so that each input is multiplied once)."""
    if isinstance(m, LatentSpec):
        rows = ((m.q_rank or m.heads * (m.dim + m.rot_dim)) + (0 if m.kv_from is not None else m.kv_rank + m.rot_dim)
                + (m.heads * m.vdim if m.gate else 0))
        out = {"w_in": (rows, hidden), "w_ukv": (m.heads * (m.dim + m.vdim), m.kv_rank), "wo": (hidden, m.heads * m.vdim)}
        if m.kv_from is None:
            out["kv_norm"] = (m.kv_rank,)
        if m.sink:
            out["sink"] = (m.heads,)
        if m.q_rank:
            out.update({"w_uq": (m.heads * (m.dim + m.rot_dim), m.q_rank), "q_norm": (m.q_rank,)})
        return out
    if isinstance(m, DeltaSpec):
        k, v = m.kv_heads * m.dim, m.heads * m.vdim
        return {"w_in": (2 * k + v + m.decay_rank + m.gate_rank + m.heads, hidden), "conv": (2 * k + v, m.conv),
                "w_a": (m.heads * m.dim, m.decay_rank), "w_g": (v, m.gate_rank), "A_log": (m.heads,), "dt_bias": (m.heads * m.dim,),
                "norm": (m.vdim,), "wo": (hidden, v)}
    if isinstance(m, AttentionSpec):
        q, k = m.heads * m.dim, m.kv_heads * m.dim
        own = k + m.kv_heads * m.vdim if m.kv_from is None else 0
        out = {"w_in": (q + own + (m.heads * m.vdim if m.gate else 0), hidden), "wo": (hidden, m.heads * m.vdim)}
        if m.distance_bias:
            out.update({"r1": (m.heads,), "r2": (m.heads,)})
        if m.qk_norm:
            out.update({"q_norm": (q,), "k_norm": (k,)})
        if m.sink:
            out["sink"] = (m.heads,)
        return out
    if isinstance(m, DifferentialSpec):
        kv = 0 if m.kv_from is not None else m.kv_heads * (2 * m.dim + m.vdim)
        out = {"w_in": (m.heads * 2 * m.dim + kv + m.heads, hidden), "q_norm": (m.dim,), "lvec": (4, m.dim), "wo": (hidden, m.heads * m.vdim)}
        if m.kv_from is None:
            out["k_norm"] = (m.dim,)
        return out
    if isinstance(m, SsmSpec):
        inner = m.heads * m.vdim
        ch = inner + 2 * m.groups * m.state
        return {"w_in": (inner + ch + m.heads, hidden), "conv": (ch, m.conv), "conv_b": (ch,), "dt_bias": (m.heads,), "A_log": (m.heads,),
                "D": (m.heads,), "norm": (inner,), "wo": (hidden, inner)}
    return {"w_in": (m.heads * 2 * (m.dim + m.vdim), hidden), "norm": (m.heads * m.vdim,), "wo": (hidden, m.heads * m.vdim)}


def expert_shapes(f: MoeSpec, hidden: int) -> dict[str, tuple]:
    """Parameter shapes of a layer's routed experts (their input projections are `w13` also where there is no gate)."""
    E = f.experts
    return {"router": (E, hidden), "bias" if f.routing is None else "correction": (E,), "w13": (E, f.up_rows, hidden), "w2": (E, hidden, f.expert.ff)}


def layer_shapes(s: LayerSpec, cfg: LayeredConfig) -> dict[str, tuple]:
    """Parameter shapes of a whole layer.  In the parallel arrangement the mixer and the dense feed-forward share their input and
    their sum, so their input projections are stacked along the rows and their output projections along the columns."""
    H = cfg.hidden_size
    mix = mixer_shapes(s.mixer, H)
    out: dict[str, tuple] = {"norm1": (H,)}
    if cfg.block == "parallel":
        ff = s.dense.ff if s.dense is not None else 0
        out["w_in"] = (mix.pop("w_in")[0] + 2 * ff, H)
        out["w_out"] = (H, mix.pop("wo")[1] + ff)
        if isinstance(s.mlp, MoeSpec):
            out.update({f"mlp.{n}": shape for n, shape in expert_shapes(s.mlp, H).items()})
    elif cfg.block == "pre_norm":
        if s.mlp is not None:
            out.update({"norm2": (H,), "mlp.w2": (H, s.mlp.ff)})
            out.update({"mlp.w13": (s.mlp.ff, H), "mlp.act": (2,)} if isinstance(s.mlp, XieluSpec) else {"mlp.w13": (2 * s.mlp.ff, H)})
        if cfg.token_side:
            out.update({"side.gate": (cfg.token_side, H), "side.proj": (H, cfg.token_side), "side.norm": (H,)})
    elif cfg.block == "two_norms":
        out["ls1"] = (H,)
        if s.mlp is not None:
            out.update({"norm2": (H,), "ls2": (H,)})
            out.update({f"mlp.{n}": shape for n, shape in expert_shapes(s.mlp, H).items()} if isinstance(s.mlp, MoeSpec) else
                       {"mlp.w13": (2 * s.mlp.ff, H), "mlp.w2": (H, s.mlp.ff)})
    else:
        out["ls1"] = (H,)
        if s.mlp is not None:
            out.update({"norm2": (H,), "ls2": (H,), "mlp.w13": (2 * s.mlp.ff, H), "mlp.w2": (H, s.mlp.ff)})
    out.update({f"mix.{n}": shape for n, shape in mix.items()})
    return out


class _Mixer(nn.Module):
    def __init__(self, spec, hidden: int, std: float, dtype, device, gen, tag: str, without: tuple = ()):
        super().__init__()
        self.spec = spec
        for name, shape in mixer_shapes(spec, hidden).items():
            if name in without:                    # projections the layer holds, stacked with others
                continue
            if len(shape) == 2:
                t = gen(f"{tag}.{name}", shape, std, dtype, device)
            else:
                t = (torch.ones if name.endswith("norm") or name == "D" else torch.zeros)(shape, dtype=dtype, device=device)
            setattr(self, name, nn.Parameter(t))


class LatentMixer(_Mixer):
    def __init__(self, spec: LatentSpec, *a):
        super().__init__(spec, *a)
        freq, self.magnitude = spec.rotary.table()
        self.register_buffer("freq", torch.tensor(freq, dtype=torch.float64, device=self.wo.device), persistent=False)
        self.layout = MX.LatentLayout(spec.heads, spec.dim, spec.rot_dim, spec.vdim, spec.kv_rank)
        # columns of the projection: queries (or their latent), latents, gate
        self.gate_at = (spec.q_rank or self.layout.q_rows) + (spec.kv_rank + spec.rot_dim if spec.kv_from is None else 0)

    def forward(self, proj, meta: ForwardMeta, run: int, eps: float):
        s = self.spec
        cache = meta.kv_cache[run if s.kv_from is None else s.kv_from][0]
        q = MX.part_norm_linear(proj[:, : s.q_rank], self.q_norm, 1, eps, self.w_uq) if s.q_rank else None
        return MX.latent_attention(proj[:, s.q_rank: self.gate_at], self.layout, cache, meta, freq=self.freq, magnitude=self.magnitude,
                                   scale=s.scale, window=s.window, sink=getattr(self, "sink", None), w_ukv=self.w_ukv,
                                   kv_norm=getattr(self, "kv_norm", None), eps=eps, q=q,
                                   gate=proj[:, self.gate_at: self.gate_at + s.heads * s.vdim] if s.gate else None)


class LinearStateMixer(_Mixer):
    def __init__(self, spec: LinearStateSpec, *a):
        super().__init__(spec, *a)
        assert len(spec.decay) == spec.heads, "one decay per head"
        self.register_buffer("decay", torch.tensor(spec.decay, dtype=torch.float64, device=self.wo.device).float(), persistent=False)

    def forward(self, proj, meta: ForwardMeta, run: int, eps: float):
        s = self.spec
        return MX.linear_state_attention(proj, s.heads, s.dim, s.vdim, self.decay, meta.states[run], meta, self.norm, eps)


class DeltaMixer(_Mixer):
    def __init__(self, spec: DeltaSpec, *a):
        super().__init__(spec, *a)
        assert spec.heads % spec.kv_heads == 0, "heads come in equal groups"
        self.layout = MX.DeltaLayout(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.conv, spec.decay_rank, spec.gate_rank)

    def forward(self, proj, meta: ForwardMeta, run: int, eps: float):
        """proj [T, q; k; v; decay latent; gate latent; β] → gated, normed outputs [T, heads · vdim]."""
        return MX.delta_rule(proj, self.layout, self.conv, self.w_a, self.w_g, self.A_log, self.dt_bias, self.norm, meta.states[run],
                             meta.states.get((run, "conv")), meta, eps)


class AttentionMixer(_Mixer):
    def __init__(self, spec: AttentionSpec, hidden: int, std: float, dtype, device, gen, tag: str, **kw):
        super().__init__(spec, hidden, std, dtype, device, gen, tag, **kw)
        assert spec.heads % spec.kv_heads == 0, "query heads come in equal groups"
        freq = spec.rotary.table()[0] if spec.rotary is not None else []
        assert 2 * len(freq) <= spec.dim, "the rotation covers at most a whole head"
        self.register_buffer("freq", torch.tensor(freq, dtype=torch.float64, device=device), persistent=False)
        self.magnitude = spec.rotary.table()[1] if spec.rotary is not None else 1.0
        assert not (spec.window and spec.chunk), "a window or chunks"
        self.layout = MX.AttentionLayout(spec.heads, spec.kv_heads, spec.dim, spec.vdim, 2 * len(freq), spec.window, spec.keep_first, spec.chunk,
                                         spec.kv_from is None, spec.value_norm)

    def forward(self, proj, meta: ForwardMeta, run: int, eps: float, out=None, aside=None):
        """proj [T, q (; k; v) (; gate; more)] → [T, heads · vdim], into `out` if given.  `aside` (mixers.Aside): what reads the same
        projection beside the attention."""
        s = self.spec
        kc, vc = meta.kv_cache[run if s.kv_from is None else s.kv_from]
        if out is None:
            out = torch.empty(proj.shape[0], s.heads * s.vdim, dtype=proj.dtype, device=proj.device)
        MX.windowed_attention(proj, self.layout, kc, vc, meta, out, freq=self.freq, magnitude=self.magnitude, scale=s.scale,
                              sink=getattr(self, "sink", None), q_norm=getattr(self, "q_norm", None), k_norm=getattr(self, "k_norm", None),
                              eps=eps, aside=aside, bias=(self.r1, self.r2) if s.distance_bias else None,
                              gate=proj[:, self.layout.rows: self.layout.rows + s.heads * s.vdim] if s.gate else None)
        return out


class DifferentialMixer(_Mixer):
    def __init__(self, spec: DifferentialSpec, hidden: int, std: float, dtype, device, gen, tag: str, **kw):
        super().__init__(spec, hidden, std, dtype, device, gen, tag, **kw)
        assert spec.heads % spec.kv_heads == 0, "query heads come in equal groups"
        self.layout = MX.DifferentialLayout(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.kv_from is None)

    def forward(self, proj, meta: ForwardMeta, run: int, eps: float, aside=None):
        """proj [T, q (; k; v); gates] → [T, heads · vdim].  `aside` (mixers.Aside): what runs beside the preparation."""
        s, t = self.spec, self.spec.temperature
        kc, vc = meta.kv_cache[run if s.kv_from is None else s.kv_from]
        return MX.differential_attention(proj, self.layout, kc, vc, meta, scale=s.scale, diff=s.diff, temperature=(t.coef, t.every) if t else None,
                                         lvec=self.lvec, q_norm=self.q_norm, k_norm=getattr(self, "k_norm", None), eps=eps, aside=aside)

    def finish(self, o, eps: float):
        return ops.linear(o, self.wo)


class SsmMixer(_Mixer):
    def __init__(self, spec: SsmSpec, hidden: int, std: float, dtype, device, gen, tag: str, **kw):
        super().__init__(spec, hidden, std, dtype, device, gen, tag, **kw)
        assert spec.heads % spec.groups == 0 and spec.heads * spec.vdim % spec.norm_groups == 0, "equal groups of heads, equal parts of a norm"
        self.layout = MX.SsmLayout(spec.heads, spec.vdim, spec.state, spec.groups, spec.conv)

    def forward(self, proj, meta: ForwardMeta, run: int, eps: float, aside=None):
        """proj [T, z; x; B; C; dt] → gated outputs [T, heads · vdim], before their norm."""
        return MX.state_space(proj, self.layout, self.conv, self.conv_b, self.dt_bias, self.A_log, self.D, meta.states[run],
                              meta.states.get((run, "conv")), meta, aside=aside)

    def finish(self, o, eps: float):
        return MX.part_norm_linear(o, self.norm, self.spec.norm_groups, eps, self.wo)


class RoutedExperts(nn.Module):
    def __init__(self, spec: MoeSpec, hidden: int, std: float, dtype, device, gen, tag: str):
        super().__init__()
        self.spec = spec
        assert 0 < spec.top <= spec.experts
        r = spec.routing
        assert r is None or (spec.experts % r.groups == 0 and 0 < r.keep <= r.groups), "experts come in equal groups"
        for name, shape in expert_shapes(spec, hidden).items():
            t = gen(f"{tag}.{name}", shape, std, dtype, device) if len(shape) > 1 else torch.zeros(shape, dtype=dtype, device=device)
            setattr(self, name, nn.Parameter(t))

    def forward(self, h, weights, index):
        """What the chosen experts of every token add (`mixers.Addend`)."""
        e = self.spec.expert
        if isinstance(e, ReluSquareSpec):
            return MX.routed_experts(h, self.w13, self.w2, weights, index, ungated=True)
        return MX.routed_experts(h, self.w13, self.w2, weights, index, e.limit, e.alpha, e.shift)


class ClampedGLU(nn.Module):
    def __init__(self, spec: GluSpec, hidden: int, std: float, dtype, device, gen, tag: str):
        super().__init__()
        self.spec = spec
        self.w13 = nn.Parameter(gen(f"{tag}.w13", (2 * spec.ff, hidden), std, dtype, device))
        self.w2 = nn.Parameter(gen(f"{tag}.w2", (hidden, spec.ff), std, dtype, device))

    def forward(self, proj):
        return ops.linear(MX.clamped_glu(proj, self.spec.limit, self.spec.alpha, self.spec.shift), self.w2)


class Xielu(nn.Module):
    def __init__(self, spec: XieluSpec, hidden: int, std: float, dtype, device, gen, tag: str):
        super().__init__()
        self.spec = spec
        self.w13 = nn.Parameter(gen(f"{tag}.w13", (spec.ff, hidden), std, dtype, device))
        self.w2 = nn.Parameter(gen(f"{tag}.w2", (hidden, spec.ff), std, dtype, device))
        self.act = nn.Parameter(torch.zeros(2, dtype=dtype, device=device))

    def forward(self, proj):
        return ops.linear(MX.xielu(proj, self.act), self.w2)


class TokenSide(nn.Module):
    """y = proj(gelu(gate x) · rows of the layer's part of a token table); the stream norms and adds it."""

    def __init__(self, dim: int, hidden: int, std: float, dtype, device, gen, tag: str):
        super().__init__()
        self.gate = nn.Parameter(gen(f"{tag}.gate", (dim, hidden), std, dtype, device))
        self.proj = nn.Parameter(gen(f"{tag}.proj", (hidden, dim), std, dtype, device))
        self.norm = nn.Parameter(torch.ones(hidden, dtype=dtype, device=device))

    def forward(self, z, tokens, table, layer: int):
        return ops.linear(MX.gelu_times_rows(z, tokens, table, layer * self.gate.shape[0]), self.proj)


class _Stream:
    """The fp32 residual and a sublayer output that has not been added to it yet.

    `project` adds the pending output (norm, layer scale, residual sum) and multiplies the new residual by a weight: one kernel
    for a handful of rows, a norm kernel and a GEMM otherwise."""

    def __init__(self, x, xb, cfg: "LayeredConfig"):
        self.x, self.xb, self.eps, self.pending = x, xb, cfg.rms_eps, None

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


MIXERS = {LatentSpec: LatentMixer, LinearStateSpec: LinearStateMixer, AttentionSpec: AttentionMixer, DifferentialSpec: DifferentialMixer,
          SsmSpec: SsmMixer, DeltaSpec: DeltaMixer}
FEED_FORWARDS = {GluSpec: ClampedGLU, XieluSpec: Xielu}


class LayeredLayer(nn.Module):
    """The "output_norm" arrangement."""

    def __init__(self, spec: LayerSpec, cfg: LayeredConfig, dtype, device, gen, layer: int):
        super().__init__()
        self.layer, self.eps = layer, cfg.rms_eps
        H, std = cfg.hidden_size, cfg.init_std

        def vec():
            return nn.Parameter(torch.ones(H, dtype=dtype, device=device))

        assert not isinstance(spec.mlp, MoeSpec), "routed experts run in the parallel arrangement"
        kind = MIXERS[type(spec.mixer)]
        self.norm1, self.ls1 = vec(), vec()
        self.mix = kind(spec.mixer, H, std, dtype, device, gen, f"L{layer}.mix")
        self.mlp = None
        if spec.mlp is not None:
            self.norm2, self.ls2 = vec(), vec()
            self.mlp = ClampedGLU(spec.mlp, H, std, dtype, device, gen, f"L{layer}.mlp")

    def forward(self, st: _Stream, meta: ForwardMeta, run: int):
        o = self.mix(st.project(self.mix.w_in), meta, run, self.eps)
        st.add(ops.linear(o, self.mix.wo), self.norm1, self.ls1)
        if self.mlp is not None:
            st.add(self.mlp(st.project(self.mlp.w13)), self.norm2, self.ls2)


class _SumStream:
    """The fp32 residual of the parallel arrangement and the sublayer outputs that have not been added to it yet.

    `project` adds them (and, before a later pass of a loop, the embedding output), norms the sum and multiplies it by the layer's
    input projection and its router: one kernel for a handful of rows; a kernel for sum and norm and the products otherwise."""

    def __init__(self, x, _copy, cfg: "LayeredConfig"):
        self.x, self.first, self.eps = x, x, cfg.rms_eps
        self.shift, self.gain = cfg.norm_shift, cfg.logit_scale
        self.pending: list = []
        self.inject = False                        # the embedding output is due before the next layer

    def _sum_into(self):
        """Where the next sum goes: never over the embedding output."""
        if not self.pending and not self.inject:
            return None
        return torch.empty_like(self.x) if self.x is self.first else self.x

    def project(self, nw, w, router=None, bias=None, want_normed: bool = False):
        """(normed residual or None, its product with `w`, fp32 router logits or None)"""
        extra = self.first if self.inject else None
        if MX.few_row_sum(self.x, self.pending, w):
            h, proj, logits, self.x = MX.sum_norm_linear(self.x, self.pending, extra, nw, self.eps, w, router, bias, want_normed)
        else:
            to = self._sum_into()
            h = MX.sum_norm(self.x, to, self.pending, extra, nw, self.eps)
            self.x = self.x if to is None else to
            proj, logits = MX.projections(h, w, router, bias)
        self.pending, self.inject = [], False
        return h, proj, logits

    def finish(self, final_w):
        # the logits' scale is part of the final norm: whatever multiplies these rows by the head sees it
        return MX.sum_norm(self.x, None, self.pending, None, final_w, self.eps, shift=self.shift, gain=self.gain)

    def value(self):
        """The residual with everything added (debugging and tests)."""
        x = torch.empty_like(self.x)
        if not self.pending:
            return x.copy_(self.x)
        MX.sum_norm(self.x, x, self.pending, None, None, self.eps)
        return x


class _TwoNormStream(_SumStream):
    """The same for the "two_norms" arrangement: sublayer outputs have scales, and the sum is normed by two weights (one root mean
    square), the second for the feed-forward's input projection or router."""

    def project(self, nw, w, nw2=None, w2=None, routes: bool = False):
        """(product of the residual normed by `nw` with `w`, product of the one normed by `nw2` with `w2` — fp32 logits where it routes,
        the normed rows of those logits)"""
        if MX.few_row_sum(self.x, self.pending, w) and (w2 is None or MX.few_row_sum(self.x, self.pending, w2)):
            proj, second, h2, self.x = MX.sum_two_norms_linear(self.x, self.pending, nw, w, nw2, w2, self.eps, self.shift, routes)
        else:
            to = self._sum_into()
            h, h2 = MX.sum_norm(self.x, to, self.pending, None, nw, self.eps, shift=self.shift, nw2=nw2, two=True)
            self.x = self.x if to is None else to
            proj = MX.product(h, w)
            second = None if w2 is None else MX.product(h2, w2, fp32=routes)
        self.pending = []
        return proj, second, h2 if routes else None


class TwoNormLayer(nn.Module):
    """The "two_norms" arrangement: x + ls1 · mixer(norm1(x)) + ls2 · feed-forward(norm2(x))."""

    def __init__(self, spec: LayerSpec, cfg: LayeredConfig, dtype, device, gen, layer: int):
        super().__init__()
        self.layer, self.eps, self.spec = layer, cfg.rms_eps, spec
        H, std, tag = cfg.hidden_size, cfg.init_std, f"L{layer}"
        assert isinstance(spec.mixer, (DifferentialSpec, SsmSpec)), "mixers of the two-norm arrangement take an aside and finish their own output"
        assert spec.dense is None or not isinstance(spec.mlp, MoeSpec), "no shared expert in the two-norm arrangement"

        def vec(value):
            return nn.Parameter(torch.full((H,), value, dtype=dtype, device=device))

        self.norm1, self.ls1 = vec(1.0 - cfg.norm_shift), vec(1.0)
        self.mix = MIXERS[type(spec.mixer)](spec.mixer, H, std, dtype, device, gen, f"{tag}.mix")
        self.mlp = None
        if spec.mlp is not None:
            self.norm2, self.ls2 = vec(1.0 - cfg.norm_shift), vec(1.0)
            self.mlp = (RoutedExperts if isinstance(spec.mlp, MoeSpec) else ClampedGLU)(spec.mlp, H, std, dtype, device, gen, f"{tag}.mlp")

    def forward(self, st: _TwoNormStream, meta: ForwardMeta, run: int):
        mlp, f = self.mlp, self.spec.mlp
        moe = isinstance(f, MoeSpec)
        if mlp is None:
            proj, second, h2 = st.project(self.norm1, self.mix.w_in)
        else:
            proj, second, h2 = st.project(self.norm1, self.mix.w_in, self.norm2, mlp.router if moe else mlp.w13, moe)
        aside = MX.Aside()
        if moe:
            aside.logits, aside.top, aside.routing, aside.correction = second, f.top, f.routing, getattr(mlp, "correction", None)
        elif mlp is not None:
            aside.glu_in, aside.glu_out = second, torch.empty(proj.shape[0], f.ff, dtype=proj.dtype, device=proj.device)
            aside.limit, aside.alpha, aside.shift = f.limit, f.alpha, f.shift
        o = self.mix(proj, meta, run, self.eps, aside=aside)
        st.pending = [MX.Addend(self.mix.finish(o, self.eps), scale=self.ls1)]
        if moe:
            if meta.record_topk is not None:
                meta.record_topk.append(_as_recorded(aside.index, meta.record_width))
            a = mlp(h2, aside.weights, aside.index)
            a.scale = self.ls2
            st.pending.append(a)
        elif mlp is not None:
            st.pending.append(MX.Addend(ops.linear(aside.glu_out, mlp.w2), scale=self.ls2))


class _PreNormStream:
    """The fp32 residual of the "pre_norm" arrangement and the sublayer output that has not been added to it yet (with its norm, if it has
    one).  `project` adds it and multiplies the new residual, normed or as it is, by a weight: one kernel for a handful of rows, a
    kernel for sum and norm and a product otherwise."""

    def __init__(self, x, _copy, cfg: LayeredConfig):
        self.x, self.eps, self.mult, self.gain = x, cfg.rms_eps, cfg.residual_mult, cfg.logit_scale
        self.pending = (None, None)

    def project(self, nw, w):
        y, yn = self.pending
        self.pending = (None, None)
        if MX.few_row_sum(self.x, (), w):
            out, self.x = MX.residual_linear(self.x, y, yn, self.mult, nw, self.eps, w)
            return out
        return MX.product(MX.residual_norm(self.x, y, yn, self.mult, nw, self.eps, w.dtype), w)

    def add(self, y, norm=None):
        self.pending = (y, norm)

    def finish(self, final_w):
        return MX.residual_norm(self.x, *self.pending, self.mult, final_w, self.eps, final_w.dtype, gain=self.gain)

    def value(self):
        """The residual with everything added (debugging and tests)."""
        x = self.x.clone()
        if self.pending[0] is not None:
            MX.residual_norm(x, *self.pending, self.mult, None, self.eps, self.pending[0].dtype)
        return x


class PreNormLayer(nn.Module):
    """The "pre_norm" arrangement: x + m · mixer(norm1(x)), then + m · feed-forward(norm2(x)), then + m · norm(token input of x)."""

    def __init__(self, spec: LayerSpec, cfg: LayeredConfig, dtype, device, gen, layer: int):
        super().__init__()
        self.layer, self.eps = layer, cfg.rms_eps
        H, std, tag = cfg.hidden_size, cfg.init_std, f"L{layer}"
        assert spec.mlp is None or type(spec.mlp) in FEED_FORWARDS, "dense feed-forwards in the pre-norm arrangement"
        assert isinstance(spec.mixer, (LatentSpec, LinearStateSpec, AttentionSpec, DeltaSpec)), "mixers that need no aside"

        def vec():
            return nn.Parameter(torch.ones(H, dtype=dtype, device=device))

        self.norm1 = vec()
        self.mix = MIXERS[type(spec.mixer)](spec.mixer, H, std, dtype, device, gen, f"{tag}.mix")
        self.mlp = self.side = None
        if spec.mlp is not None:
            self.norm2 = vec()
            self.mlp = FEED_FORWARDS[type(spec.mlp)](spec.mlp, H, std, dtype, device, gen, f"{tag}.mlp")
        if cfg.token_side:
            self.side = TokenSide(cfg.token_side, H, std, dtype, device, gen, f"{tag}.side")

    def forward(self, st: _PreNormStream, meta: ForwardMeta, run: int):
        o = self.mix(st.project(self.norm1, self.mix.w_in), meta, run, self.eps)
        st.add(ops.linear(o, self.mix.wo))
        if self.mlp is not None:
            st.add(self.mlp(st.project(self.norm2, self.mlp.w13)))
        if self.side is not None:
            st.add(self.side(st.project(None, self.side.gate), *st.token_rows, self.layer), self.side.norm)


class ParallelLayer(nn.Module):
    """The "parallel" arrangement: x + mixer(norm(x)) + feed-forward(norm(x)).

    One input projection feeds queries, keys, values and the dense feed-forward; one output projection multiplies the concatenation
    of the heads' outputs and the dense activations, so their sum is part of the product.  Routed experts run beside it."""

    def __init__(self, spec: LayerSpec, cfg: LayeredConfig, dtype, device, gen, layer: int):
        super().__init__()
        self.layer, self.eps, self.dense = layer, cfg.rms_eps, spec.dense
        H, std, tag = cfg.hidden_size, cfg.init_std, f"L{layer}"
        assert isinstance(spec.mixer, AttentionSpec), "the parallel arrangement is built for attention mixers"
        assert spec.mlp is None or (isinstance(spec.mlp, MoeSpec) and spec.mlp.routing is None) or spec.dense is not None
        shapes = layer_shapes(spec, cfg)
        self.norm1 = nn.Parameter(torch.ones(H, dtype=dtype, device=device))
        self.w_in = nn.Parameter(gen(f"{tag}.w_in", shapes["w_in"], std, dtype, device))
        self.w_out = nn.Parameter(gen(f"{tag}.w_out", shapes["w_out"], std, dtype, device))
        self.mix = MIXERS[type(spec.mixer)](spec.mixer, H, std, dtype, device, gen, f"{tag}.mix", without=("w_in", "wo"))
        self.mlp = RoutedExperts(spec.mlp, H, std, dtype, device, gen, f"{tag}.mlp") if isinstance(spec.mlp, MoeSpec) else None
        self.at_dense = mixer_shapes(spec.mixer, H)["w_in"][0]      # first row of the dense feed-forward in the projection
        self.mix_out = spec.mixer.heads * spec.mixer.vdim

    def forward(self, st: _SumStream, meta: ForwardMeta, run: int):
        moe = self.mlp
        h, proj, logits = st.project(self.norm1, self.w_in, *((moe.router, moe.bias, True) if moe is not None else ()))
        both = torch.empty(proj.shape[0], self.w_out.shape[1], dtype=proj.dtype, device=proj.device)
        aside = MX.Aside(logits=logits, top=moe.spec.top if moe is not None else 0)
        if self.dense is not None:
            aside.glu_in, aside.glu_out = proj[:, self.at_dense:], both[:, self.mix_out:]
            aside.limit, aside.alpha, aside.shift = self.dense.limit, self.dense.alpha, self.dense.shift
        self.mix(proj, meta, run, self.eps, out=both[:, : self.mix_out], aside=aside)
        st.pending = [MX.Addend(ops.linear(both, self.w_out))]
        if moe is not None:
            if meta.record_topk is not None:
                meta.record_topk.append(_as_recorded(aside.index, meta.record_width))
            st.pending.append(moe(h, aside.weights, aside.index))


def _as_recorded(index, width: int):
    """Expert ids of one layer in the width the engine records (−1: no such choice)."""
    if index.shape[1] == width:
        return index
    return torch.nn.functional.pad(index, (0, width - index.shape[1]), value=-1)


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
        assert cfg.block in BLOCKS, f"unknown arrangement of layers '{cfg.block}'"
        for i, s in enumerate(cfg.layer_specs):
            m = s.mixer
            if isinstance(m, LatentSpec) and m.kv_from is not None:
                src = cfg.layer_specs[m.kv_from].mixer
                assert m.kv_from < i and isinstance(src, LatentSpec) and src.kv_from is None and (src.kv_rank, src.rot_dim) == (
                    m.kv_rank, m.rot_dim), f"layer {i} cannot read the latents of layer {m.kv_from}"
            if isinstance(m, (DifferentialSpec, AttentionSpec)) and m.kv_from is not None:
                src = cfg.layer_specs[m.kv_from].mixer
                assert m.kv_from < i and type(src) is type(m) and src.kv_from is None and (src.kv_heads, src.dim, src.vdim) == (
                    m.kv_heads, m.dim, m.vdim), f"layer {i} cannot read the keys and values of layer {m.kv_from}"
        assert cfg.norm_shift == 0.0 or cfg.block == "two_norms", "norm weights stored around another value: two-norm arrangement only"
        assert (cfg.residual_mult == 1.0 and not cfg.token_side) or cfg.block == "pre_norm", "residual factor, token input: pre-norm arrangement only"
        assert cfg.logit_scale == 1.0 or cfg.block != "output_norm", "a logit scale is part of the final norm of the summing streams"
        if cfg.loop is not None:
            assert 0 <= cfg.loop.start < cfg.loop.stop <= cfg.num_layers and cfg.loop.times > 0, f"{cfg.loop} of {cfg.num_layers} layers"
            assert cfg.block == "parallel", "loops are built for the parallel arrangement"
        kind = BLOCKS[cfg.block][0]
        self.layers = nn.ModuleList(kind(s, cfg, dtype, device, gen, l) for l, s in enumerate(cfg.layer_specs))
        self.runs = cfg.runs()
        self.bigram = None
        if cfg.bigram is not None:
            self.bigram = nn.Parameter(gen("bigram", (cfg.bigram.buckets + 1, cfg.hidden_size), cfg.init_std, dtype, device))
        self.side_embed = None
        if cfg.token_side:
            self.side_embed = nn.Parameter(gen("side_embed", (cfg.vocab_size, cfg.num_layers * cfg.token_side), cfg.init_std, dtype, device))
        self.num_moe_layers = cfg.num_moe_layers
        if cfg.norm_shift:
            with torch.no_grad():
                self.norm.fill_(1.0 - cfg.norm_shift)
        H = cfg.hidden_size
        freq = [cfg.position_base ** (-2.0 * i / H) for i in range((H + 1) // 2)] if cfg.position_base else []
        self.register_buffer("position_freq", torch.tensor(freq, dtype=torch.float64, device=device) if freq else None, persistent=False)

    # ---- what the engine keeps per token and per sequence ------------------------------------------------------------
    def _run_mixers(self):
        return [(r, self.layers[l].mix) for r, (l, _) in enumerate(self.runs)]

    def kv_rows(self) -> dict[int, tuple]:
        """Cache row shapes per token of every layer run that writes one."""
        rows: dict[int, tuple] = {}
        for r, m in self._run_mixers():
            if isinstance(m, LatentMixer) and m.spec.kv_from is None:
                rows[r] = ((m.layout.pitch,),)
            elif isinstance(m, AttentionMixer) and m.spec.kv_from is None:
                rows[r] = ((m.spec.kv_heads, m.spec.dim), (m.spec.kv_heads, m.spec.vdim))
            elif isinstance(m, DifferentialMixer) and m.spec.kv_from is None:
                rows[r] = ((m.spec.kv_heads, 2 * m.spec.dim), (m.spec.kv_heads, m.spec.vdim))      # a key row holds both maps
        return rows

    def state_shapes(self) -> dict:
        """fp32 state per sequence of every recurrent layer run; under (run, "conv") the last inputs of its convolution."""
        out: dict = {}
        for r, m in self._run_mixers():
            if isinstance(m, LinearStateMixer):
                out[r] = (m.spec.heads, m.spec.dim, m.spec.vdim)
            elif isinstance(m, SsmMixer):
                out[r] = (m.spec.heads, m.spec.state, m.spec.vdim)
            elif isinstance(m, DeltaMixer):
                out[r] = (m.spec.heads, m.spec.dim, m.spec.vdim)
            if isinstance(m, (SsmMixer, DeltaMixer)) and m.spec.conv > 1:
                out[(r, "conv")] = (m.spec.conv, m.layout.channels)
        return out

    def forward(self, tokens, meta: ForwardMeta, hidden_in=None, inputs_embeds=None):
        if torch.is_grad_enabled():
            raise NotImplementedError("layered models run in the engine only: no backward pass is built for their mixers")
        assert meta.ragged is not None, "layered models take ragged engine batches"
        big = self.cfg.bigram
        st = BLOCKS[self.cfg.block][1](*MX.bigram_embedding(tokens, meta.prev_tokens, self.embed, self.bigram,
                                                            (big.buckets, big.mul_prev, big.mul_cur) if big is not None else None,
                                                            want_copy=self.cfg.block == "output_norm", positions=meta.positions,
                                                            freq=self.position_freq), self.cfg)
        st.token_rows = (tokens, self.side_embed)
        meta.record_width = self.cfg.moe_topk
        for run, (l, inject) in enumerate(self.runs):
            st.inject = inject
            self.layers[l](st, meta, run)
            if meta.record_residual is not None:
                meta.record_residual.append(st.value())
        return st.finish(self.norm)

    def logits(self, hidden):
        lg = super().logits(hidden)
        return MX.softcap_(lg, self.cfg.logit_softcap, exact=self.embed.dtype == torch.float32) if self.cfg.logit_softcap else lg

    def log_probs(self, hidden, targets, temperature: float = 1.0, with_entropy: bool = False):
        if not self.cfg.logit_softcap:
            return super().log_probs(hidden, targets, temperature, with_entropy)
        out, entropy = [], []
        for h, t in zip(hidden.split(512), targets.split(512)):        # a few rows of the whole vocabulary at a time
            lp = torch.log_softmax(self.logits(h).float() / temperature, -1)
            out.append(lp.gather(-1, t.long()[:, None]).squeeze(-1))
            if with_entropy:
                entropy.append(-(lp.exp() * lp).sum(-1))
        return torch.cat(out), torch.cat(entropy) if with_entropy else None


# arrangement → (layer, stream of residual and pending outputs)
BLOCKS = {"output_norm": (LayeredLayer, _Stream), "parallel": (ParallelLayer, _SumStream), "two_norms": (TwoNormLayer, _TwoNormStream),
          "pre_norm": (PreNormLayer, _PreNormStream)}
