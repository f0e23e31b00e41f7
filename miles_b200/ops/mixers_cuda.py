"""CUDA execution of the ops in `mixers.py` (inference only): the kernels of mixers.cu, latent_attn.cu and linear_state.cu.

Tensors are bf16, or float32 throughout (then every product is a true 32-bit one: the kernels' own fp32 loops, and cuBLAS
without TF32 for the dense projections, as `ops.linear` does for float32).
"""
from __future__ import annotations

import torch

from .cuda import C, gemm_nt


def _c(x):
    return x if x.is_contiguous() else x.contiguous()


def bigram_embedding(tokens, prev, embed, table, spec):
    T, D = tokens.numel(), embed.shape[1]
    x = torch.empty(T, D, dtype=torch.float32, device=embed.device)
    xb = torch.empty(T, D, dtype=embed.dtype, device=embed.device)
    buckets, mp, mc = spec if table is not None else (0, 0, 0)
    C.bigram_embedding(tokens.to(torch.int32), prev, embed, table, buckets, mp, mc, x, xb)
    return x, xb


def output_norm_residual(x, y, nw, ls, eps, final_w=None):
    xb = torch.empty_like(y)
    C.output_norm(x, _c(y), nw, ls, final_w, xb, float(eps))
    return x, xb


def few_row_projection(y, w) -> bool:
    return False


def clamped_glu(h, limit, alpha):
    out = torch.empty(h.shape[0], h.shape[1] // 2, dtype=h.dtype, device=h.device)
    C.clamped_glu(_c(h), out, float(limit), float(alpha))
    return out


def gated_norm(o, w, gate, eps):
    out = torch.empty_like(o)
    C.gated_norm(o, w, gate, out, float(eps))
    return out


def linear_state(proj, H, dk, dv, decay, state, meta):
    out = torch.empty(proj.shape[0], H * dv, dtype=proj.dtype, device=proj.device)
    C.linear_state(proj, decay, state, meta.state_slots, meta.ragged.cu_q, meta.positions, out)
    return out


def latent_attention(proj, lay, cache, meta, freq, magnitude, scale, window, sink, w_ukv, kv_norm, eps):
    T, H = proj.shape[0], lay.heads
    sizes = [H, lay.dim, lay.rot, lay.vdim, lay.rank, lay.rank_p, lay.pitch]
    dt, dev = proj.dtype, proj.device
    t_long = 0
    q_abs = torch.empty(T - t_long, H, lay.pitch, dtype=dt, device=dev)
    C.latent_prep(proj, meta.positions, meta.slot_mapping, freq, float(magnitude), kv_norm, float(eps), cache, q_abs, None, t_long, 0, 0, sizes)
    w_uk = w_ukv[: H * lay.dim].view(H, lay.dim, lay.rank)
    w_uv = w_ukv[H * lay.dim:].view(H, lay.vdim, lay.rank)
    out = torch.empty(T, H, lay.vdim, dtype=dt, device=dev)
    q_nope = proj[t_long:, : lay.q_rows].unflatten(1, (H, lay.dim + lay.rot))[..., : lay.dim]
    C.head_linear(q_nope, w_uk, False, q_abs[..., : lay.rank])
    o_lat = torch.empty(T - t_long, H, lay.rank, dtype=dt, device=dev)
    seq = meta.ragged.token_seq
    C.latent_attend(q_abs, cache, meta.block_table, seq[t_long:] if seq is not None else None, meta.positions[t_long:], meta.slot_mapping[t_long:],
                    sink, o_lat, float(scale), int(window), sizes)
    C.head_linear(o_lat, w_uv, True, out[t_long:])
    return out.view(T, H * lay.vdim)
