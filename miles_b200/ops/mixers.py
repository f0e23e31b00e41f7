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

    @property
    def rows(self) -> int:
        return self.heads * self.dim + self.kv_heads * (self.dim + self.vdim)


@dataclass
class Addend:
    """A sublayer's output on its way into the residual: rows `y` [T, D], or (with `dst`) the expert-sorted rows `y` whose sum
    Σ_j weights[t, j] · y[dst[t, j]] is meant."""

    y: torch.Tensor
    weights: torch.Tensor | None = None
    dst: torch.Tensor | None = None


@dataclass
class Aside:
    """Work on the same projection that runs beside an attention layer's preparation: the choice of experts from `logits`
    (→ `weights`, `index`) and the activation of a dense feed-forward (`glu_in` [T, ≥ 2F] → `glu_out` [T, F], both may be strided)."""

    logits: torch.Tensor | None = None
    top: int = 0
    weights: torch.Tensor | None = None
    index: torch.Tensor | None = None
    glu_in: torch.Tensor | None = None
    glu_out: torch.Tensor | None = None
    limit: float = 0.0
    alpha: float = 0.0


def bigram_embedding(tokens, prev, embed, table=None, spec=None, want_copy=True):
    """(fp32 residual, copy in the model's dtype or None): embed[token] + table[(prev·m_prev + token·m_cur) mod buckets]; a sequence's first
    token (prev < 0) takes the table's last row.  spec = (buckets, m_prev, m_cur)."""
    if embed.is_cuda:
        return _k().bigram_embedding(tokens, prev, embed, table, spec, want_copy)
    return ref.bigram_embedding(tokens, prev, embed, table, spec)


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


def clamped_glu(h, limit, alpha):
    """h = [gate; up] → g·sigmoid(alpha·g)·(u + 1), g = min(gate, limit), u = clamp(up, ±limit)."""
    if h.is_cuda:
        return _k().clamped_glu(h, limit, alpha)
    return ref.clamped_glu(h, limit, alpha)


def latent_attention(proj, lay: LatentLayout, cache, meta, *, freq, magnitude, scale, window, sink, w_ukv, kv_norm, eps):
    """proj [T, q rows (+ rank + rot)] → attention output [T, heads·vdim].  Rotates queries and (with `kv_norm`) norms, rotates
    and caches the new latents; then every token attends to the cached latents it sees."""
    if proj.is_cuda:
        return _k().latent_attention(proj, lay, cache, meta, freq, magnitude, scale, window, sink, w_ukv, kv_norm, eps)
    return ref.latent_attention(proj, lay, cache, meta, freq, magnitude, scale, window, sink, w_ukv, kv_norm, eps)


def linear_state_attention(proj, heads, dk, dv, decay, state, meta, norm_w, eps):
    """proj = [q; k; v; gate] of every token → rmsnorm(all heads' outputs)·norm_w·sigmoid(gate), with silu(q), silu(k), silu(v) and
    per head S ← decay·S + k vᵀ, o = Sᵀ q.  `state` [slots, heads, dk, dv] fp32 is read (zero at position 0) and written."""
    gate = proj[:, heads * (2 * dk + dv):]
    if proj.is_cuda:
        o = _k().linear_state(proj, heads, dk, dv, decay, state, meta)
        return _k().gated_norm(o, norm_w, gate, eps)
    return ref.gated_norm(ref.linear_state(proj, heads, dk, dv, decay, state, meta), norm_w, gate, eps)


def sum_norm(x, to, addends, extra, nw, eps):
    """s = x + Σ addends (+ extra), fp32, written to `to` if given; returns rmsnorm(s)·nw in the model's dtype (None without `nw`)."""
    if x.is_cuda:
        return _k().sum_norm(x, to, addends, extra, nw, eps)
    return ref.sum_norm(x, to, addends, extra, nw, eps)


def few_row_sum(x, addends, w) -> bool:
    return x.is_cuda and _k().few_row_sum(x, addends, w)


def sum_norm_linear(x, addends, extra, nw, eps, w, w2=None, b2=None, want_normed=False):
    """`sum_norm` and `projections` in one kernel (where `few_row_sum` holds).  Returns (normed or None, product, logits, sum)."""
    return _k().sum_norm_linear(x, addends, extra, nw, eps, w, w2, b2, want_normed)


def projections(h, w, w2=None, b2=None):
    """(h·wᵀ in the model's dtype, fp32 h·w2ᵀ + b2 or None)."""
    if h.is_cuda:
        return _k().projections(h, w, w2, b2)
    return ref.projections(h, w, w2, b2)


def windowed_attention(proj, lay: AttentionLayout, kc, vc, meta, out, *, freq, magnitude, scale, sink, q_norm, k_norm, eps, aside=None):
    """proj [T, ≥ q; k; v] → `out` [T, heads·vdim] (may be strided).  Norms queries and keys over the whole projection, rotates them,
    caches keys and values; then every token attends to the cached tokens it sees: those less than `window` back, and the first
    `keep` ones.  `aside` is done on the way."""
    if proj.is_cuda:
        return _k().windowed_attention(proj, lay, kc, vc, meta, out, freq, magnitude, scale, sink, q_norm, k_norm, eps, aside)
    if aside is not None:
        if aside.logits is not None:
            aside.weights, aside.index = ref.topk_softmax(aside.logits, aside.top)
        if aside.glu_in is not None:
            aside.glu_out.copy_(ref.clamped_glu(aside.glu_in[:, : 2 * aside.glu_out.shape[1]], aside.limit, aside.alpha))
    return ref.windowed_attention(proj, lay, kc, vc, meta, out, freq, magnitude, scale, sink, q_norm, k_norm, eps)


def routed_experts(h, w13, w2, weights, index, limit, alpha) -> Addend:
    """Σ_j weights[t, j] · W2[e]·clamped_glu(W13[e]·h[t]) with e = index[t, j], as an addend."""
    if h.is_cuda:
        return _k().routed_experts(h, w13, w2, weights, index, limit, alpha)
    return Addend(ref.routed_experts(h, w13, w2, weights, index, limit, alpha))
