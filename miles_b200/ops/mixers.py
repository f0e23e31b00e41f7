"""Ops of the layer-by-layer decoders (models/layered.py): CUDA tensors run `mixers_cuda.py` (the sm_100a extension), CPU tensors
the statements in `mixers_reference.py`."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from . import mixers_reference as ref

_cuda = None


def _k():
    global _cuda
    if _cuda is None:
        from . import mixers_cuda as _c

        _cuda = _c
    return _cuda


def _up16(n: int) -> int:
    return (n + 15) // 16 * 16


@dataclass(frozen=True)
class LatentLayout:
    """Sizes of one latent-attention layer.  A cached row is [latent | zeros to a multiple of 16 | rotated key part | zeros to a
    multiple of 16]: both parts are whole tensor-core steps and every row starts on a 16-byte boundary."""

    heads: int
    dim: int
    rot: int
    vdim: int
    rank: int

    @property
    def q_rows(self) -> int:
        return self.heads * (self.dim + self.rot)

    @property
    def rank_p(self) -> int:
        return _up16(self.rank)

    @property
    def pitch(self) -> int:
        return self.rank_p + _up16(self.rot)


@dataclass(frozen=True)
class AttentionLayout:
    """Sizes of one grouped-query attention layer; the cache keeps [kv_heads, dim] keys and [kv_heads, vdim] values per token."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot: int           # rotated dimensions of a head, the first ones
    window: int        # 0: no window
    keep: int          # first tokens a window keeps
    chunk: int = 0     # 0: no chunks
    writes: bool = True            # the layer has keys and values of its own
    value_norm: bool = False       # they are kept with every head's values over their root mean square

    @property
    def rows(self) -> int:
        return self.heads * self.dim + (self.kv_heads * (self.dim + self.vdim) if self.writes else 0)


@dataclass(frozen=True)
class DeltaLayout:
    """Sizes of one gated-delta-rule layer; a row of its projection is [q | k | v | decay latent | gate latent | β]."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int
    gate_rank: int

    @property
    def key_rows(self) -> int:
        return self.kv_heads * self.dim

    @property
    def channels(self) -> int:
        """q, k and v: what passes the convolution."""
        return 2 * self.key_rows + self.heads * self.vdim

    @property
    def gate_at(self) -> int:
        return self.channels + self.decay_rank

    @property
    def beta_at(self) -> int:
        return self.gate_at + self.gate_rank


@dataclass(frozen=True)
class DifferentialLayout:
    """Sizes of one differential-attention layer.  The cache keeps [kv_heads, 2·dim] keys (both maps side by side) and [kv_heads, vdim]
    values per token; `writes`: the layer has keys and values of its own."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    writes: bool = True

    @property
    def q_rows(self) -> int:
        return self.heads * 2 * self.dim

    @property
    def gate_at(self) -> int:
        return self.q_rows + (self.kv_heads * (2 * self.dim + self.vdim) if self.writes else 0)

    @property
    def paired(self) -> AttentionLayout:
        """The grouped-query layer it is to the attention kernels: every map a query head over whole key rows."""
        return AttentionLayout(2 * self.heads, self.kv_heads, 2 * self.dim, self.vdim, 0, 0, 0)


@dataclass(frozen=True)
class SsmLayout:
    """Sizes of one state-space layer; a row of its projection is [z | x | B | C | dt]."""

    heads: int
    vdim: int
    state: int
    groups: int
    taps: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """x, B and C: what passes the convolution."""
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class Routing:
    """Choice of experts by sigmoid scores: corrected scores compete inside the `keep` best of `groups` groups of neighbours (a group is
    worth its two largest); weights are the chosen ones' uncorrected scores over their sum, times `scale`."""

    groups: int = 1
    keep: int = 1
    scale: float = 1.0


@dataclass
class Addend:
    """A sublayer's output on its way into the residual: rows `y` [T, D], or (with `dst`) the expert-sorted rows `y` whose sum
    Σ_j weights[t, j] · y[dst[t, j]] is meant."""

    y: torch.Tensor
    weights: torch.Tensor | None = None
    dst: torch.Tensor | None = None
    scale: torch.Tensor | None = None      # a factor per channel


@dataclass
class Aside:
    """Work that runs beside a mixer's preparation: the choice of experts from `logits` (→ `weights`, `index`; by `routing` and
    `correction` if given, else by a softmax over the largest) and the activation of a dense feed-forward (`glu_in` [T, ≥ 2F] →
    `glu_out` [T, F], both may be strided)."""

    logits: torch.Tensor | None = None
    top: int = 0
    weights: torch.Tensor | None = None
    index: torch.Tensor | None = None
    glu_in: torch.Tensor | None = None
    glu_out: torch.Tensor | None = None
    limit: float = 0.0
    alpha: float = 0.0
    shift: float = 1.0
    routing: Routing | None = None
    correction: torch.Tensor | None = None


def bigram_embedding(tokens, prev, embed, table=None, spec=None, want_copy=True, positions=None, freq=None):
    """(fp32 residual, copy in the model's dtype or None): embed[token] + table[(prev·m_prev + token·m_cur) mod buckets]; a sequence's first
    token (prev < 0) takes the table's last row.  spec = (buckets, m_prev, m_cur).  `freq` (one per pair of channels): the sine and the
    cosine of position · freq are added to the pair."""
    if embed.is_cuda:
        return _k().bigram_embedding(tokens, prev, embed, table, spec, want_copy, positions, freq)
    return ref.bigram_embedding(tokens, prev, embed, table, spec, positions, freq)


def output_norm_residual(x, y, nw, ls, eps, final_w=None):
    """x ← x + rmsnorm(y)·nw·ls (fp32, in place).  Returns (x, its copy in y's dtype), the copy RMS-normed with `final_w` if given."""
    if x.is_cuda:
        return _k().output_norm_residual(x, y, nw, ls, eps, final_w)
    return ref.output_norm_residual(x, y, nw, ls, eps, final_w)


def few_row_projection(y, w) -> bool:
    return y.is_cuda and _k().few_row_projection(y, w)


def output_norm_linear(x, y, nw, ls, eps, w):
    """(x', x'·wᵀ) with x' = x + rmsnorm(y)·nw·ls in one kernel (where `few_row_projection` holds).  Returns (product, x')."""
    return _k().output_norm_linear(x, y, nw, ls, eps, w)


def clamped_glu(h, limit, alpha, shift=1.0):
    """h = [gate; up] → g·sigmoid(alpha·g)·(u + shift), g = min(gate, limit), u = clamp(up, ±limit)."""
    if h.is_cuda:
        return _k().clamped_glu(h, limit, alpha, shift)
    return ref.clamped_glu(h, limit, alpha, shift)


def latent_attention(proj, lay: LatentLayout, cache, meta, *, freq, magnitude, scale, window, sink, w_ukv, kv_norm, eps, q=None, gate=None):
    """proj [T, q rows (+ rank + rot)], or q [T, q rows] and proj [T, (rank + rot)] → attention output [T, heads·vdim], times
    sigmoid(gate) if given.  Rotates queries and (with `kv_norm`) norms, rotates and caches the new latents; then every token attends
    to the cached latents it sees."""
    kv = proj[:, lay.q_rows:] if q is None else proj
    q = proj[:, : lay.q_rows] if q is None else q
    f = _k().latent_attention if proj.is_cuda else ref.latent_attention
    return f(q, kv, lay, cache, meta, freq, magnitude, scale, window, sink, w_ukv, kv_norm, eps, gate)


def linear_state_attention(proj, heads, dk, dv, decay, state, meta, norm_w, eps):
    """proj = [q; k; v; gate] of every token → rmsnorm(all heads' outputs)·norm_w·sigmoid(gate), with silu(q), silu(k), silu(v) and
    per head S ← decay·S + k vᵀ, o = Sᵀ q.  `state` [slots, heads, dk, dv] fp32 is read (zero at position 0) and written."""
    gate = proj[:, heads * (2 * dk + dv):]
    if proj.is_cuda:
        o = _k().linear_state(proj, heads, dk, dv, decay, state, meta)
        return _k().gated_norm(o, norm_w, gate, eps)
    return ref.gated_norm(ref.linear_state(proj, heads, dk, dv, decay, state, meta), norm_w, gate, eps)


def sum_norm(x, to, addends, extra, nw, eps, shift=0.0, gain=1.0, nw2=None, two=False):
    """s = x + Σ addends (+ extra), fp32, written to `to` if given; returns rmsnorm(s)·(nw + shift)·gain in the model's dtype (None without
    `nw`); with `two` a pair, the second by `nw2` (None without)."""
    h = (_k() if x.is_cuda else ref).sum_norm(x, to, addends, extra, nw, eps, shift, gain, nw2)
    return h if two else h[0]


def few_row_sum(x, addends, w) -> bool:
    return x.is_cuda and _k().few_row_sum(x, addends, w)


def sum_norm_linear(x, addends, extra, nw, eps, w, w2=None, b2=None, want_normed=False):
    """`sum_norm` and `projections` in one kernel (where `few_row_sum` holds).  Returns (normed or None, product, logits, sum)."""
    return _k().sum_norm_linear(x, addends, extra, nw, eps, w, w2, b2, want_normed)


def sum_two_norms_linear(x, addends, nw, w, nw2, w2, eps, shift, routes):
    """Sum, two norms of it and the product of each with its weight in one kernel (where `few_row_sum` holds for both weights; `w2` may be
    None).  Returns (first product, second product — fp32 where it `routes`, the rows normed by `nw2` there, sum)."""
    return _k().sum_two_norms_linear(x, addends, nw, w, nw2, w2, eps, shift, routes)


def product(h, w, fp32=False):
    """h·wᵀ in the model's dtype or fp32; rows may be padded to whole 16-byte pieces."""
    if h.is_cuda:
        return _k().product(h, w, fp32)
    y = h @ w.T
    return y.float() if fp32 else y


def projections(h, w, w2=None, b2=None):
    """(h·wᵀ in the model's dtype, fp32 h·w2ᵀ + b2 or None)."""
    if h.is_cuda:
        return _k().projections(h, w, w2, b2)
    return ref.projections(h, w, w2, b2)


def windowed_attention(proj, lay: AttentionLayout, kc, vc, meta, out, *, freq, magnitude, scale, sink, q_norm, k_norm, eps, aside=None, bias=None,
                       gate=None):
    """proj [T, ≥ q (; k; v)] → `out` [T, heads·vdim] (may be strided).  Norms queries and keys over the whole projection, rotates them,
    caches keys and values (those of a layer that has its own); then every token attends to the cached tokens it sees: those less than
    `window` back, and the first `keep` ones, or those of its own `chunk`.  `bias` (r1, r2 per head): r1·ln(1 + r2·distance) off the
    scores; `gate` [T, heads·vdim]: outputs times its sigmoid.  `aside` is done on the way."""
    if proj.is_cuda:
        return _k().windowed_attention(proj, lay, kc, vc, meta, out, freq, magnitude, scale, sink, q_norm, k_norm, eps, aside, bias, gate)
    ref.aside(aside)
    return ref.windowed_attention(proj, lay, kc, vc, meta, out, freq, magnitude, scale, sink, q_norm, k_norm, eps, bias, gate)


def delta_rule(proj, lay: DeltaLayout, conv, w_a, w_g, A_log, dt_bias, norm_w, state, ring, meta, eps):
    """proj [T, q; k; v; decay latent; gate latent; β] → [T, heads·vdim].  Causal convolution and silu on q, k, v; q and k to unit vectors per
    head (q over √dim on top); decays g = exp(−exp(A_log)·softplus(w_a·latent + dt_bias)) per head and key channel; per head
    S ← diag(g)·S, S ← S + k (σ(β)·(v − Sᵀk))ᵀ, o = Sᵀq; every head's o over its root mean square, times norm_w and the sigmoid of w_g·latent.
    `state` [slots, heads, dim, vdim] and `ring` [slots, taps, channels] (the convolution's inputs by position mod taps; None
    without look-back), fp32, are read (nothing before position 0) and written."""
    f = _k().delta_rule if proj.is_cuda else ref.delta_rule
    return f(proj, lay, conv, w_a, w_g, A_log, dt_bias, norm_w, state, ring, meta, eps)


def residual_norm(x, y, yn, mult, nw, eps, dtype, gain=1.0):
    """x ← x + mult·y, or x + mult·rmsnorm(y)·yn (fp32, in place; y None: x as it is).  Returns rmsnorm(x)·nw·gain in `dtype` (without
    `nw`: a copy of x)."""
    return (_k() if x.is_cuda else ref).residual_norm(x, y, yn, mult, nw, eps, dtype, gain)


def residual_linear(x, y, yn, mult, nw, eps, w):
    """`residual_norm` and the product with w in one kernel (where `few_row_sum` holds).  Returns (product, new x)."""
    return _k().residual_linear(x, y, yn, mult, nw, eps, w)


def xielu(z, act):
    """z²·softplus(act₀) + z/2 for z > 0, (½ + softplus(act₁))·(exp(z) − 1 − z) + z/2 for z ≤ 0."""
    return (_k() if z.is_cuda else ref).xielu(z, act)


def gelu_times_rows(z, tokens, table, col):
    """gelu(z) (tanh form) times columns [col, col + width) of the tokens' rows of `table`."""
    return (_k() if z.is_cuda else ref).gelu_times_rows(z, tokens, table, col)


def softcap_(logits, cap, exact=False):
    """logits ← cap·tanh(logits / cap), fp32 in place; `exact`: good to 32 bits."""
    return (_k() if logits.is_cuda else ref).softcap_(logits, cap, exact)


def differential_attention(proj, lay: DifferentialLayout, kc, vc, meta, *, scale, diff, temperature, lvec, q_norm, k_norm, eps, aside=None):
    """proj [T, q (; k; v); gates] → [T, heads·vdim].  Norms queries and keys per head and map, multiplies queries by the temperature
    (coef, every) of their position, caches keys and values (with `k_norm`; else they are another layer's); every token attends to all
    cached tokens up to itself with both maps of every head: o = a1 − λ·a2 with λ = exp(l₀·l₁) − exp(l₂·l₃) + diff (rows of `lvec`),
    normed over the head, times (1 − diff) · sigmoid(gate of the head).  `aside` is done on the way."""
    if proj.is_cuda:
        return _k().differential_attention(proj, lay, kc, vc, meta, scale, diff, temperature, lvec, q_norm, k_norm, eps, aside)
    ref.aside(aside)
    return ref.differential_attention(proj, lay, kc, vc, meta, scale, diff, temperature, lvec, q_norm, k_norm, eps)


def state_space(proj, lay: SsmLayout, conv, conv_b, dt_bias, A_log, D, state, ring, meta, aside=None):
    """proj [T, z; x; B; C; dt] → [T, heads·vdim] = y·silu(z): causal convolution and silu on x, B, C; dt ← softplus(dt + dt_bias); per head
    S ← exp(−exp(A_log)·dt)·S + dt·B xᵀ, y = Sᵀ C + D·x.  `state` [slots, heads, state, vdim] and `ring` [slots, taps, channels] (the
    convolution's inputs by position mod taps; None without look-back), fp32, are read (nothing before position 0) and written.  `aside` is done on the way."""
    if proj.is_cuda:
        return _k().state_space(proj, lay, conv, conv_b, dt_bias, A_log, D, state, ring, meta, aside)
    ref.aside(aside)
    return ref.state_space(proj, lay, conv, conv_b, dt_bias, A_log, D, state, ring, meta)


def part_norm_linear(x, nw, parts, eps, w):
    """(every one of `parts` equal parts of a row over its own root mean square, times nw)·wᵀ"""
    if x.is_cuda:
        return _k().part_norm_linear(x, nw, parts, eps, w)
    return ref.part_norm(x, nw, parts, eps) @ w.T


def routed_experts(h, w13, w2, weights, index, limit=0.0, alpha=0.0, shift=1.0, ungated=False) -> Addend:
    """Σ_j weights[t, j] · W2[e]·act(W13[e]·h[t]) with e = index[t, j], as an addend; act: `clamped_glu`, or relu(·)² without a gate."""
    if h.is_cuda:
        return _k().routed_experts(h, w13, w2, weights, index, limit, alpha, shift, ungated)
    return Addend(ref.routed_experts(h, w13, w2, weights, index, limit, alpha, shift, ungated))
