"""CUDA execution of the ops in `mixers.py` (inference only): the kernels of mixers.cu, latent_*.cu, linear_*.cu, window_*.cu,
diff_prep.cu, ssm_*.cu, delta_*.cu, attention_*_tc.cu, paged_attend.cu and experts_any.cu.

Tensors are bf16, or float32 throughout (then every product is a true 32-bit one: the kernels' own fp32 loops, and cuBLAS
without TF32 for the dense projections, as `ops.linear` does for float32).
"""
from __future__ import annotations

import os

import torch

from . import cuda as K
from .cuda import BF16, C, GEMV_MAX_N, gemv_ok


def _c(x):
    return x if x.is_contiguous() else x.contiguous()


def bigram_embedding(tokens, prev, embed, table, spec, want_copy=True, positions=None, freq=None):
    T, D = tokens.numel(), embed.shape[1]
    x = torch.empty(T, D, dtype=torch.float32, device=embed.device)
    xb = torch.empty(T, D, dtype=embed.dtype, device=embed.device) if want_copy else None
    buckets, mp, mc = spec if table is not None else (0, 0, 0)
    C.bigram_embedding(tokens.to(torch.int32), prev, embed, table, buckets, mp, mc, positions if freq is not None else None, freq, x, xb)
    return x, xb


def output_norm_residual(x, y, nw, ls, eps, final_w=None):
    xb = torch.empty_like(y)
    C.output_norm(x, _c(y), nw, ls, final_w, xb, float(eps))
    return x, xb


# rows up to which the output norm runs inside the projection that follows it (every CTA of that projection repeats the norm)
FUSED_NORM_M = int(os.environ.get("MILES_OUTPUT_NORM_GEMV_M", "4"))


def few_row_projection(y, w) -> bool:
    return y.shape[0] <= FUSED_NORM_M and w.shape[0] <= GEMV_MAX_N and gemv_ok(y, w)


def output_norm_linear(x, y, nw, ls, eps, w):
    out = torch.empty(y.shape[0], w.shape[0], dtype=y.dtype, device=y.device)
    x_new = torch.empty_like(x)
    C.gemv_output_norm(x, _c(y), nw, ls, float(eps), w, out, x_new, bool(w.is_leaf and w.requires_grad))
    return out, x_new


def clamped_glu(h, limit, alpha, shift=1.0):
    out = torch.empty(h.shape[0], h.shape[1] // 2, dtype=h.dtype, device=h.device)
    C.clamped_glu(h, out, float(limit), float(alpha), shift=float(shift))
    return out


def gated_norm(o, w, gate, eps):
    out = torch.empty_like(o)
    C.gated_norm(o, w, gate, out, float(eps))
    return out


def linear_state(proj, H, dk, dv, decay, state, meta):
    out = torch.empty(proj.shape[0], H * dv, dtype=proj.dtype, device=proj.device)
    rg, slots, cu_q = meta.ragged, meta.state_slots, meta.ragged.cu_q
    if rg.n_long and proj.dtype == BF16 and dk % 8 == 0 and dv % 8 == 0 and dk <= 128 and dv <= 128 and proj.stride(0) % 8 == 0:
        # long pieces in chunks on the tensor cores, the short ones behind them token by token
        segs, seq_segs, multi = _segments(meta, H)
        seg_state = torch.empty(segs.shape[0], H, dk, dv, dtype=torch.float32, device=proj.device) if multi else None
        C.linear_chunk(proj, decay, state, slots, meta.positions, segs, seq_segs, seg_state, out)
        if slots.numel() == rg.n_long:
            return out
        slots, cu_q = slots[rg.n_long:], cu_q[rg.n_long:]
    C.linear_state(proj, decay, state, slots, cu_q, meta.positions, out)
    return out


def _segment_cost(chunks: list[int], c: int, H: int, sms: int = 148) -> float:
    """Chunk times of segments of c chunks: waves of full segments, the shorter last ones beside or behind the last wave.  A CTA's
    start counts as one and a half chunks.  (A cut costs its caller a pass over keys and values more.)"""
    start = 1.5
    full, rest = sum(n // c for n in chunks) * H, [n % c for n in chunks if n % c]
    waves = -(-full // sms)
    time, slots = waves * (c + start), waves * sms - full
    if rest:
        if not slots:
            return time + -(-len(rest) * H // sms) * (max(rest) + start)
        time = max(time, (waves - 1) * (c + start) + -(-len(rest) * H // slots) * (max(rest) + start))
    return time


def _segments(meta, H: int):
    """Cut the long pieces of a batch into segments of whole 64-token chunks so that the (segment, head) CTAs, one per SM at a time,
    finish in the fewest chunk times.  Returns ([n, 4] (sequence, first token, end, last of its sequence), offsets per sequence, any
    sequence cut)."""
    rg = meta.ragged
    key = ("segments", H)
    if key not in rg.scratch:
        lens = rg.q_lens[: rg.n_long]
        whole = -(-max(lens) // 64)                     # chunks of the longest piece
        size = 64 * min((_segment_cost([-(-n // 64) for n in lens], c, H) * (1.0 if c >= whole else 1.4), c) for c in {*range(2, 17), whole})[1]
        segs, cu, t = [], [0], 0
        for b, n in enumerate(lens):
            for a in range(0, n, size):
                segs += [b, t + a, t + min(n, a + size), int(a + size >= n)]
            t += n
            cu.append(len(segs) // 4)
        d = torch.tensor(segs + cu, dtype=torch.int32).to(meta.positions.device)
        rg.scratch[key] = (d[: len(segs)].view(-1, 4), d[len(segs):], len(segs) // 4 > rg.n_long)
    return rg.scratch[key]


# bf16 sizes the tensor-core kernels take; anything else runs the any-size kernels of latent_attn.cu
def _mma_ok(lay, dt) -> bool:
    return dt == BF16 and lay.dim % 8 == 0 and lay.vdim % 8 == 0 and lay.rank % 8 == 0 and lay.rot % 8 == 0 and lay.rank_p <= 512 and lay.pitch <= 640


def _prefill_ok(lay, dt, scale) -> bool:
    return _mma_ok(lay, dt) and lay.dim <= 128 and lay.rot <= 64 and lay.vdim <= 128 and scale > 0


def decode_splits(tokens: int, heads: int, window: int, block_size: int) -> int:
    """Key splits of latent_decode: enough (token, head group, split) CTAs for the 148 SMs (one resident per SM), whole key tiles."""
    group = 32 if block_size % 64 == 0 or heads > 16 else 16
    return max(1, min(32, 148 // (tokens * -(-heads // group)), -(-(window or 4096) // 64)))


def _key_ranges(meta, window: int):
    """Keys the long pieces of a batch can see: packed offsets [n + 1] and first position per sequence (device), and their number."""
    rg = meta.ragged
    if window not in rg.scratch:
        base = [max(0, s - q - window + 1) if window else 0 for s, q in zip(rg.seq_lens[: rg.n_long], rg.q_lens)]
        cu = [0]
        for s, b in zip(rg.seq_lens, base):
            cu.append(cu[-1] + s - b)
        t = torch.tensor(cu + base, dtype=torch.int32).to(meta.positions.device)
        rg.scratch[window] = (t[: len(cu)], t[len(cu):], cu[-1], max(rg.q_lens[: rg.n_long]))
    return rg.scratch[window]


def _head_linear(x, w, w_nk, y, fast, gate=None):
    (C.head_linear_mma if fast else C.head_linear)(x, w, w_nk, y, gate)


def _whole_rows(x):
    """Rows that start on 16-byte boundaries: x itself, or a copy in rows of whole 16-byte pieces (None stays None)."""
    piece = 16 // x.element_size() if x is not None else 1
    if x is None or (x.stride(0) % piece == 0 and x.data_ptr() % 16 == 0):
        return x
    return _rows(x.shape[0], x.shape[1], x.dtype, x.device).copy_(x)


def latent_attention(q, kv, lay, cache, meta, freq, magnitude, scale, window, sink, w_ukv, kv_norm, eps, gate=None):
    T, H, rg = q.shape[0], lay.heads, meta.ragged
    sizes = [H, lay.dim, lay.rot, lay.vdim, lay.rank, lay.rank_p, lay.pitch]
    dt, dev = q.dtype, q.device
    fast = _mma_ok(lay, dt)
    t_long = rg.t_long if _prefill_ok(lay, dt, scale) else 0
    n_short = T - t_long
    q_nope = (lay.dim + 63) // 64 * 64
    q_abs = torch.empty(n_short, H, lay.pitch, dtype=dt, device=dev)
    q_full = torch.empty(t_long, H, q_nope + 64, dtype=dt, device=dev)
    C.latent_prep(q, kv, meta.positions, meta.slot_mapping, freq, float(magnitude), kv_norm, float(eps), cache, q_abs, q_full, t_long, q_nope,
                  q_nope + 64, sizes)
    out = torch.empty(T, H, lay.vdim, dtype=dt, device=dev)
    if n_short:
        w_uk, w_uv = w_ukv[: H * lay.dim].view(H, lay.dim, lay.rank), w_ukv[H * lay.dim:].view(H, lay.vdim, lay.rank)
        qn = q[t_long:].unflatten(1, (H, lay.dim + lay.rot))[..., : lay.dim]
        aligned = fast and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0
        _head_linear(qn, w_uk, False, q_abs[..., : lay.rank], aligned)
        o_lat = torch.empty(n_short, H, lay.rank, dtype=dt, device=dev)
        seq = rg.token_seq[t_long:] if rg.token_seq is not None else None
        pos, slots = meta.positions[t_long:], meta.slot_mapping[t_long:]
        if fast:
            splits = decode_splits(n_short, H, window, cache.shape[1])
            part_o = torch.empty(n_short * H * splits * lay.rank_p, dtype=torch.float32, device=dev)
            part_ml = torch.empty(n_short * H * splits * 2, dtype=torch.float32, device=dev)
            C.latent_decode(q_abs, cache, meta.block_table, seq, pos, slots, sink, part_o, part_ml, o_lat, float(scale), int(window), splits, sizes,
                            C.error_flag(q))
        else:
            C.latent_attend(q_abs, cache, meta.block_table, seq, pos, slots, sink, o_lat, float(scale), int(window), sizes)
        _head_linear(o_lat, w_uv, True, out[t_long:], fast, gate[t_long:] if gate is not None else None)
    if t_long:
        cu_k, base, total, max_q = _key_ranges(meta, window)
        lat = torch.empty(total, lay.pitch, dtype=dt, device=dev)
        C.latent_gather(cache, meta.block_table, cu_k, base, lat)
        N = H * (lay.dim + lay.vdim)
        kv = torch.empty(total, N, dtype=dt, device=dev)
        C.gemm(lat, w_ukv, kv, total, N, lay.rank, lay.pitch, lay.rank, N, False, False, False, None, 0)
        C.latent_prefill(q_full, kv, lat, out, sink, rg.cu_q, cu_k, rg.n_long, max_q, float(scale), int(window), sizes, C.error_flag(q),
                         _whole_rows(gate[:t_long]) if gate is not None else None)
    return out.view(T, H * lay.vdim)


# ---- parallel arrangement: sum, norm, projections ---------------------------------------------------------------------

def _split_addends(addends):
    """(two dense outputs or None, expert-sorted rows or None) for one kernel."""
    dense = [a.y for a in addends if a.dst is None]
    rows = [a for a in addends if a.dst is not None]
    assert len(dense) <= 2 and len(rows) <= 1, "a sum takes two dense outputs and one set of experts' rows"
    return dense + [None] * (2 - len(dense)), (rows[0] if rows else None)


def sum_norm(x, to, addends, extra, nw, eps, shift=0.0, gain=1.0, nw2=None):
    (y1, y2), r = _split_addends(addends)
    h, h2 = (torch.empty(x.shape, dtype=w.dtype, device=x.device) if w is not None else None for w in (nw, nw2))
    s1, s2 = _scales(addends)
    C.sum_norm(x, to, y1, s1, y2, s2, r.y if r else None, r.weights if r else None, r.dst if r else None, extra, nw, h, nw2, h2, float(eps),
               float(shift), float(gain))
    return h, h2


def _scales(addends):
    """Scales of the first dense output and of what comes with it (another dense output, else experts' rows)."""
    dense, rows = [a.scale for a in addends if a.dst is None], [a.scale for a in addends if a.dst is not None]
    second = dense[1:] + rows
    return dense[0] if dense else None, second[0] if second else None


def few_row_sum(x, addends, w) -> bool:
    return (w.dtype == BF16 and x.shape[0] <= FUSED_NORM_M and w.shape[0] <= GEMV_MAX_N and K._gemv_k_ok(x.shape[0], w.shape[1])
            and all(a.dst is None for a in addends))


def _static(w) -> bool:
    return bool(w.is_leaf and w.requires_grad)


def sum_norm_linear(x, addends, extra, nw, eps, w, w2, b2, want_normed):
    (y1, y2), _ = _split_addends(addends)
    T, dev = x.shape[0], x.device
    proj = torch.empty(T, w.shape[0], dtype=w.dtype, device=dev)
    logits = torch.empty(T, w2.shape[0], dtype=torch.float32, device=dev) if w2 is not None else None
    x_new = torch.empty_like(x) if addends or extra is not None else None
    h = torch.empty(x.shape, dtype=w.dtype, device=dev) if want_normed else None
    C.gemv_sum_norm(x, y1, None, y2, None, extra, None, nw, None, float(eps), 0.0, w, proj, w2, b2, logits, x_new, h, _static(w))
    return h, proj, logits, x if x_new is None else x_new


def _rows(T: int, n: int, dtype, device):
    """[T, n] in rows of whole 16-byte pieces, so that kernels behind a projection of any width can use them."""
    piece = 16 // torch.empty(0, dtype=dtype).element_size()
    return torch.empty(T, -(-n // piece) * piece, dtype=dtype, device=device)[:, :n]


def sum_two_norms_linear(x, addends, nw, w, nw2, w2, eps, shift, routes):
    (y1, y2), _ = _split_addends(addends)
    s1, s2 = _scales(addends)
    T, dev = x.shape[0], x.device
    proj = _rows(T, w.shape[0], w.dtype, dev)
    second = None
    if w2 is not None:
        second = torch.empty(T, w2.shape[0], dtype=torch.float32, device=dev) if routes else _rows(T, w2.shape[0], w.dtype, dev)
    x_new = torch.empty_like(x) if addends else None
    h2 = torch.empty(x.shape, dtype=w.dtype, device=dev) if routes else None
    C.gemv_sum_norm(x, y1, s1, y2, s2, None, None, nw, nw2, float(eps), float(shift), w, proj, w2, None, second, x_new, h2,
                    _static(w) and (w2 is None or _static(w2)))
    return proj, second, h2, x if x_new is None else x_new


def product(h, w, fp32):
    if h.dtype != BF16:
        return torch.nn.functional.linear(h, w)
    if fp32:
        return K.gemm_nt(h, w, out_dtype=torch.float32)
    return K.gemm_nt(h, w, _rows(h.shape[0], w.shape[0], BF16, h.device))


def projections(h, w, w2, b2):
    if h.dtype != BF16:
        logits = None if w2 is None else torch.addmm(b2, h, w2.t())
        return torch.nn.functional.linear(h, w), logits
    T, E = h.shape[0], w2.shape[0] if w2 is not None else 0
    if w2 is not None and T <= K.GEMV_M and w.shape[0] <= GEMV_MAX_N and gemv_ok(h, w):
        proj = torch.empty(T, w.shape[0], dtype=BF16, device=h.device)
        logits = torch.empty(T, E, dtype=torch.float32, device=h.device)
        C.gemv_sum_norm(None, None, None, None, None, None, h, None, None, 0.0, 0.0, w, proj, w2, b2, logits, None, None, _static(w))
        return proj, logits
    return K.gemm_nt(h, w), None if w2 is None else K.gemm_nt(h, w2, bias=b2, out_dtype=torch.float32)


# ---- windowed grouped-query attention ---------------------------------------------------------------------------------

def _window_ok(lay, dt) -> bool:
    """Sizes the tensor-core kernels take; anything else runs paged_attend.cu."""
    return dt == BF16 and lay.dim % 8 == 0 and lay.vdim % 8 == 0 and lay.dim <= 128 and lay.vdim <= 128


def window_splits(tokens: int, lay) -> int:
    """CTAs of a cluster that share the keys of one (token, key head): enough for the SMs, at most one per tile of 64 keys."""
    group = lay.heads // lay.kv_heads
    ctas = tokens * lay.kv_heads * -(-group // (16 if group > 8 else 8))
    tiles = -(-(lay.window + lay.keep) // 64) if lay.window else -(-lay.chunk // 64) if lay.chunk else 64
    return max(1, min(8, tiles, 444 // ctas))


def windowed_attention(proj, lay, kc, vc, meta, out, freq, magnitude, scale, sink, q_norm, k_norm, eps, aside, bias=None, gate=None):
    T, rg, dt, dev = proj.shape[0], meta.ragged, proj.dtype, proj.device
    fast = _window_ok(lay, dt) and out.stride(0) % 8 == 0
    pitch = -(-lay.dim // 64) * 64 if fast else lay.dim
    sizes = [lay.heads, lay.kv_heads, lay.dim, lay.vdim, lay.rot, lay.window, lay.keep, pitch, lay.chunk]
    q = torch.empty(T, lay.heads, pitch, dtype=dt, device=dev)
    C.window_prep(proj, meta.positions, meta.slot_mapping, freq, float(magnitude), q_norm, k_norm, float(eps), kc if lay.writes else None,
                  vc if lay.writes else None, q, sizes, *_aside(aside, T), lay.value_norm)
    _paged_attention(q, lay, kc, vc, meta, out, scale, sink, sizes, fast, bias=bias, gate=_whole_rows(gate) if fast else gate)


def _aside(a, T: int):
    """The arguments of a kernel that does an `Aside` on the way; allocates what it chooses."""
    if a is None:
        return [None] * 6, [0.0] * 4, [0] * 3
    if a.logits is not None:
        a.weights = torch.empty(T, a.top, dtype=torch.float32, device=a.logits.device)
        a.index = torch.empty(T, a.top, dtype=torch.int32, device=a.logits.device)
    r = a.routing
    return ([a.logits, a.weights if a.logits is not None else None, a.index if a.logits is not None else None, a.glu_in, a.glu_out, a.correction],
            [float(a.limit), float(a.alpha), float(a.shift), float(r.scale) if r else 1.0], [1, r.groups, r.keep] if r else [0, 1, 1])


def _paged_attention(q, lay, kc, vc, meta, out, scale, sink, sizes, fast, difference=(), bias=None, gate=None):
    """Prepared queries over the paged cache: long pieces as query tiles, short ones token by token.  `difference`: (weight of the second map,
    gates, gain, eps) of differential attention; `bias` (r1, r2), `gate`: see `windowed_attention`."""
    T, rg = q.shape[0], meta.ragged
    r1, r2 = bias or (None, None)
    t_long = rg.t_long if fast and scale > 0 and kc.shape[1] % 8 == 0 and lay.heads // lay.kv_heads <= 128 else 0
    if t_long:
        C.window_prefill(q, kc, vc, out, sink, rg.cu_q, meta.positions, meta.block_table, rg.n_long, max(rg.q_lens[: rg.n_long]), t_long,
                         float(scale), sizes, C.error_flag(q), *difference, r1=r1, r2=r2, out_gate=gate)
    if T > t_long:
        seq = rg.token_seq[t_long:] if rg.token_seq is not None else None
        where = (kc, vc, meta.block_table, seq, meta.positions[t_long:], meta.slot_mapping[t_long:], sink)
        extra = dict(r1=r1, r2=r2, out_gate=gate[t_long:] if gate is not None else None)
        if difference:
            difference = (difference[0], difference[1][t_long:], *difference[2:])
        if fast:
            C.window_decode(q[t_long:], *where, out[t_long:], float(scale), window_splits(T - t_long, lay), sizes, *difference, **extra)
        elif difference:
            both = torch.empty(T - t_long, lay.heads * lay.vdim, dtype=torch.float32, device=q.device)
            C.window_attend(q[t_long:], *where, both, float(scale), sizes)
            C.diff_combine(both, out[t_long:], lay.heads // 2, lay.vdim, *difference)
        else:
            C.window_attend(q[t_long:], *where, out[t_long:], float(scale), sizes, **extra)


def differential_attention(proj, lay, kc, vc, meta, scale, diff, temperature, lvec, q_norm, k_norm, eps, aside):
    T, dt, dev, pair = proj.shape[0], proj.dtype, proj.device, lay.paired
    out = torch.empty(T, lay.heads * lay.vdim, dtype=dt, device=dev)
    fast = _window_ok(pair, dt)
    pitch = -(-pair.dim // 64) * 64 if fast else pair.dim
    sizes = [pair.heads, pair.kv_heads, pair.dim, pair.vdim, 0, 0, 0, pitch]
    q = torch.empty(T, pair.heads, pitch, dtype=dt, device=dev)
    lam = torch.empty(1, dtype=torch.float32, device=dev)
    coef, every = temperature or (0.0, 1.0)
    C.diff_prep(proj, meta.positions, meta.slot_mapping, q_norm, k_norm, lvec, lam, kc if lay.writes else None, vc if lay.writes else None, q,
                [lay.heads, lay.kv_heads if lay.writes else 0, lay.dim, lay.vdim, pitch], float(eps), float(coef), float(every), float(diff),
                *_aside(aside, T))
    gates = proj[:, lay.gate_at: lay.gate_at + lay.heads]
    _paged_attention(q, pair, kc, vc, meta, out, scale, None, sizes, fast, (lam, gates, 1.0 - diff, float(eps)))
    return out


# ---- gated delta rule -------------------------------------------------------------------------------------------------

def _low_rank(x, w, x2, w2):
    """(x·wᵀ, x2·w2ᵀ) for rows that are part of a wider projection."""
    if x.dtype != BF16:
        return torch.nn.functional.linear(x, w), torch.nn.functional.linear(x2, w2)
    T = x.shape[0]

    def aligned(a):
        return a.stride(0) % 8 == 0 and a.data_ptr() % 16 == 0

    if T <= K.GEMV_M and x.shape[1] == x2.shape[1] and aligned(x) and aligned(x2) and K._gemv_k_ok(T, x.shape[1]) and max(w.shape[0], w2.shape[0]) <= GEMV_MAX_N:
        y, y2 = (torch.empty(T, m.shape[0], dtype=BF16, device=x.device) for m in (w, w2))
        C.gemv_sum_norm(None, None, None, None, None, None, x, None, None, 0.0, 0.0, w, y, w2, None, y2, None, None, _static(w) and _static(w2), x2=x2)
        return y, y2

    def one(a, m):
        n = a.shape[1]
        if T <= K.GEMV_M or n % 8 or not aligned(a):
            return K.gemm_nt(a.clone(memory_format=torch.contiguous_format), m)      # (a single row counts as contiguous wherever it starts)
        out = _rows(T, m.shape[0], BF16, a.device)
        C.gemm(a, m, out, T, m.shape[0], n, a.stride(0), n, out.stride(0), False, False, False, None, 0)
        return out

    return one(x, w), one(x2, w2)


def delta_rule(proj, lay, conv, w_a, w_g, A_log, dt_bias, norm_w, state, ring, meta, eps):
    T, dt, dev, rg = proj.shape[0], proj.dtype, proj.device, meta.ragged
    sizes = [lay.heads, lay.kv_heads, lay.dim, lay.vdim, lay.taps, lay.beta_at]
    raw, gate = _low_rank(proj[:, lay.channels: lay.gate_at], w_a, proj[:, lay.gate_at: lay.beta_at], w_g)
    out = torch.empty(T, lay.heads * lay.vdim, dtype=dt, device=dev)

    def tensors(slots, positions, raw):
        return [conv, A_log, dt_bias, state, ring, slots, positions, raw]

    slots, cu_q = meta.state_slots, rg.cu_q
    if cu_q is None and C.delta_step_ok(lay.dim, lay.vdim):
        C.delta_step(proj, sizes, tensors(slots, meta.positions, raw), norm_w, gate, float(eps), out)
        return out
    act = torch.empty(T, lay.channels, dtype=dt, device=dev)
    C.delta_conv(proj, sizes, tensors(slots, meta.positions, raw), _conv_tiles(meta, lay.taps) if cu_q is not None else None, cu_q, act)
    n = rg.n_long if dt == BF16 and lay.dim % 8 == 0 and lay.vdim % 8 == 0 and lay.dim <= 128 and lay.vdim <= 128 and cu_q is not None else 0
    if n:                                # long pieces in chunks on the tensor cores, the short ones behind them token by token
        err = C.error_flag(proj)
        for chunks, parts in _chunk_rounds(meta, lay):
            scratch = torch.empty(chunks.shape[0] * lay.heads * C.delta_chunk_bytes(lay.dim, lay.vdim), dtype=torch.uint8, device=dev)
            C.delta_chunk(proj, act, sizes, tensors(slots, meta.positions, raw), chunks, parts, scratch, scan_warps(parts.shape[0] * lay.heads, lay.vdim),
                          out, err)
    if slots.numel() > n:
        C.delta_seq(proj, act, sizes, tensors(slots[n:], meta.positions, raw), cu_q[n:] if cu_q is not None else None, out)
    normed = torch.empty_like(out)
    C.head_gated_norm(out, norm_w, gate, normed, float(eps))
    return normed


DELTA_SCRATCH = int(os.environ.get("MILES_DELTA_SCRATCH_MB", "800")) << 20      # what a round of chunks leaves for its second kernel, at most


def _chunk_rounds(meta, lay):
    """The long pieces of a batch in chunks of 64 tokens, in rounds whose scratch stays within bounds; in each every piece gets its share, and
    its state passes through its slot.  Returns [(chunks [n, 4], parts [n, 4])] (see mb_delta_chunk)."""
    rg = meta.ragged
    key = ("delta", lay.heads, lay.dim, lay.vdim)
    if key not in rg.scratch:
        lens = rg.q_lens[: rg.n_long]
        whole = sum(-(-n // 64) for n in lens)
        rounds = -(-whole // max(1, min(65535, DELTA_SCRATCH // (lay.heads * C.delta_chunk_bytes(lay.dim, lay.vdim)))))
        tables = []
        for r in range(rounds):
            chunks, parts, t = [], [], 0
            for b, n in enumerate(lens):
                per = -(-(-(-n // 64)) // rounds) * 64
                lo, hi = min(n, r * per), min(n, (r + 1) * per)
                if lo < hi:
                    parts += [len(chunks) // 4, -(-(hi - lo) // 64), b, 0]
                    for a in range(lo, hi, 64):
                        chunks += [b, t + a, t + min(hi, a + 64), 0]
                t += n
            if chunks:
                d = torch.tensor(chunks + parts, dtype=torch.int32).to(meta.positions.device)
                tables.append((d[: len(chunks)].view(-1, 4), d[len(chunks):].view(-1, 4)))
        rg.scratch[key] = tables
    return rg.scratch[key]


def scan_warps(pairs: int, vdim: int, sms: int = 148) -> int:
    """Warps of a CTA of delta_chunk's second kernel, 16 value columns each: the fewest waves of CTAs (one per SM), each slower the more warps
    share the SM."""
    slices = -(-vdim // 16)
    return min((-(-pairs * -(-slices // w) // sms) * cost, w) for w, cost in ((8, 1.0), (4, 0.6), (2, 0.45)) if w == 2 or w <= slices)[1]


# ---- state-space mixer ------------------------------------------------------------------------------------------------

def _conv_tiles(meta, taps: int):
    """[n, 4] (first token, end, sequence, first tile of its piece) over all pieces of a packed batch.  A tile has at least as many tokens as the
    convolution looks back (ssm_state.cu)."""
    rg = meta.ragged
    T = sum(rg.q_lens)
    size = max(32 if T > 4096 else 16, taps - 1)
    if ("conv tiles", size) not in rg.scratch:
        tiles, t = [], 0
        for b, n in enumerate(rg.q_lens):
            for a in range(0, n, size):
                tiles += [t + a, t + min(n, a + size), b, int(a == 0)]
            t += n
        rg.scratch["conv tiles", size] = torch.tensor(tiles, dtype=torch.int32).to(meta.positions.device).view(-1, 4)
    return rg.scratch["conv tiles", size]


def state_space(proj, lay, conv, conv_b, dt_bias, A_log, D, state, ring, meta, aside):
    T, dt, dev, rg = proj.shape[0], proj.dtype, proj.device, meta.ragged
    sizes = [lay.heads, lay.vdim, lay.state, lay.groups, lay.taps]
    out = torch.empty(T, lay.inner, dtype=dt, device=dev)
    a = _aside(aside, T)

    def tensors(slots, positions):
        return [conv, conv_b, dt_bias, A_log, D, state, ring, slots, positions]

    slots, cu_q = meta.state_slots, rg.cu_q
    if cu_q is None and lay.vdim % 4 == 0 and lay.vdim <= 1024 and lay.state <= 4096:
        C.ssm_step(proj, sizes, tensors(slots, meta.positions), out, *a)
        return out
    xbc = torch.empty(T, lay.channels, dtype=dt, device=dev)
    step, decay = (torch.empty(T, lay.heads, dtype=torch.float32, device=dev) for _ in range(2))
    C.ssm_conv(proj, sizes, tensors(slots, meta.positions), _conv_tiles(meta, lay.taps) if cu_q is not None else None, cu_q, xbc, step, decay, *a)
    if rg.n_long and dt == BF16 and lay.state % 8 == 0 and lay.vdim % 8 == 0 and lay.state <= 128 and lay.vdim <= 128 and proj.stride(0) % 2 == 0:
        # long pieces in chunks on the tensor cores, the short ones behind them token by token
        segs, seq_segs, multi = _segments(meta, lay.heads // C.ssm_heads_per_cta(lay.heads, lay.vdim, lay.groups))
        seg_state = torch.empty(segs.shape[0], lay.heads, lay.state, lay.vdim, dtype=torch.float32, device=dev) if multi else None
        seg_decay = torch.empty(segs.shape[0], lay.heads, dtype=torch.float32, device=dev) if multi else None
        C.ssm_chunk(proj, xbc, step, decay, sizes, tensors(slots, meta.positions), segs, seq_segs, seg_state, seg_decay, out)
        if slots.numel() == rg.n_long:
            return out
        slots, cu_q = slots[rg.n_long:], cu_q[rg.n_long:]
    C.ssm_seq(proj, xbc, step, decay, sizes, tensors(slots, meta.positions), cu_q, out)
    return out


def residual_norm(x, y, yn, mult, nw, eps, dtype, gain=1.0):
    h = torch.empty(x.shape, dtype=dtype, device=x.device)
    if yn is None:
        C.sum_norm(x, x if y is not None else None, y, None, None, None, None, None, None, None, nw, h, None, None, float(eps), 0.0, float(gain), float(mult))
    else:
        C.output_norm(x, _c(y), yn, None, nw, h, float(eps), float(mult), float(gain))
    return h


def residual_linear(x, y, yn, mult, nw, eps, w):
    out = _rows(x.shape[0], w.shape[0], w.dtype, x.device)
    if y is None:
        C.gemv_sum_norm(x, None, None, None, None, None, None, nw, None, float(eps), 0.0, w, out, None, None, None, None, None, _static(w))
        return out, x
    x_new = torch.empty_like(x)
    if yn is None:
        C.gemv_sum_norm(x, _c(y), None, None, None, None, None, nw, None, float(eps), 0.0, w, out, None, None, None, x_new, None, _static(w), float(mult))
    else:
        C.gemv_output_norm(x, _c(y), yn, None, float(eps), w, out, x_new, _static(w), float(mult), nw)
    return out, x_new


def xielu(z, act):
    z = _c(z)
    out = torch.empty_like(z)
    C.xielu(z, act, out)
    return out


def gelu_times_rows(z, tokens, table, col):
    out = torch.empty(z.shape, dtype=z.dtype, device=z.device)
    C.gelu_rows(z, tokens.to(torch.int32), table, col, out)
    return out


def softcap_(logits, cap, exact):
    C.softcap(logits, float(cap), bool(exact))
    return logits


def part_norm_linear(x, nw, parts, eps, w):
    if parts == 1 and w.shape[0] <= GEMV_MAX_N and gemv_ok(x, w) and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0:
        y = torch.empty(x.shape[0], w.shape[0], dtype=BF16, device=x.device)
        C.gemv(x, None, nw, float(eps), w, None, y, None, None, _static(w))      # a handful of rows: the norm inside the product
        return y
    h = torch.empty(x.shape, dtype=x.dtype, device=x.device)
    C.part_norm(x, nw, h, parts, float(eps))
    return K.linear(h, w)


# ---- routed experts ---------------------------------------------------------------------------------------------------

def routed_experts(h, w13, w2, weights, index, limit, alpha, shift=1.0, ungated=False):
    from . import cuda_more as M
    from .mixers import Addend

    T, k = index.shape
    E, rows, D = w13.shape
    F = w2.shape[2]
    glu = (0.0, 0.0, 0.0) if ungated else (float(limit), float(alpha), float(shift))
    if M.few_token_experts(h, w13, T, k, ungated):
        act = torch.empty(T * k, F, dtype=BF16, device=h.device)
        out = torch.empty_like(h)
        C.moe_gemv(h, w13, w2, index, weights, act, out, 0, *glu, ungated)
        return Addend(out)
    if h.dtype == BF16 and D % 8 == 0 and F % 8 == 0 and k <= 64 and E <= 2048:
        bt = M.small_moe_bt(T * k, E, w13, w2)
        x_perm, seg, tile, dst = M.sort_by_expert(h, index, E, bt)
        return Addend(M.experts_forward(x_perm, w13, w2, seg, tile, bt, "relu2" if ungated else glu)[1], weights, dst)
    act = torch.empty(T * k, F, dtype=h.dtype, device=h.device)
    out = torch.empty_like(h)
    C.experts_any(h, w13, w2, index, weights, act, out, *glu)
    return Addend(out)
