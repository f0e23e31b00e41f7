"""Ops of the layer-by-layer decoders (models/layered.py): CUDA tensors run `mixers_cuda.py` (the sm_100a extension), CPU tensors
the statements in `mixers_reference.py`."""
from __future__ import annotations

from dataclasses import dataclass

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


def bigram_embedding(tokens, prev, embed, table=None, spec=None):
    """(fp32 residual, copy in the model's dtype): embed[token] + table[(prev·m_prev + token·m_cur) mod buckets]; a sequence's first
    token (prev < 0) takes the table's last row.  spec = (buckets, m_prev, m_cur)."""
    if embed.is_cuda:
        return _k().bigram_embedding(tokens, prev, embed, table, spec)
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
