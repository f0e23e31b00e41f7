"""Prefill and decode of a layer-by-layer decoder beside the closest other model of equal width, depth and feed-forward.

    python bench.py --layered [--layered-model NAME] [--layered-baseline NAME] [--layers N]

NAME: nopelorn-4B-shape, ronupel-30B-A3B-shape, vozirax-30B-A3B-shape or senadra-4B-shape.

The baseline is qwen3-4B for a dense model and qwen3-30B-A3B for one with routed experts, with as many layers as the layered model has
layer runs; nopelorn-4B-shape (latent and linear attention) for a model with delta-rule layers.

Random weights, synthetic tokens.  `throughput`: whole models through the engine (device-timed forwards and decode graphs).
`kernels`: the mixers' kernels one by one at the same sizes with their distance from the measured roofline, next to the kernels
of the grouped-query model that do the like work.  L2 is flushed between timed kernel launches; model forwards move far more
bytes than L2 holds.
"""
from __future__ import annotations

import json
import os

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))


def peaks() -> tuple[float, float, str]:
    """(bytes/s, bf16 FLOP/s, which): the measured copy bandwidth and GEMM rate of this machine if recorded, else fallbacks."""
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "measured"
    except (OSError, KeyError):
        return 6.65e12, 1.59e15, "fallback"


class _Timer:
    def __init__(self):
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def ms(self, fn, iters: int = 10, warmup: int = 3) -> float:
        for _ in range(warmup):
            fn()
        total = 0.0
        for _ in range(iters):
            self.flush.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            total += e0.elapsed_time(e1)
        return total / iters


@torch.no_grad()
def throughput(cfg, prefill=((1, 8192), (8, 1024)), decode=((1, 2048), (8, 2048), (64, 2048)), iters: int = 5) -> dict:
    """Tokens/s of prefill batches (sequences × length) and decode steps (rows × context), device-timed."""
    g = torch.Generator().manual_seed(0)
    rows = max([n for n, _ in prefill] + [n for n, _ in decode])
    ctx = max([l for _, l in prefill] + [l + 64 for _, l in decode])
    ctx_tokens = max([n * l for n, l in prefill] + [n * (l + 64) for n, l in decode])
    from .engine import Engine

    eng = Engine(cfg, device="cuda:0", dtype=torch.bfloat16, num_blocks=ctx_tokens // 64 + 2 * rows, block_size=64, max_running_requests=rows,
                 max_context_len=ctx, prefix_cache=False)
    out: dict = {"model": cfg.name, "layers": cfg.num_layers, "params": cfg.num_params(), "prefill": [], "decode": []}

    def opened(n, length):
        reqs = []
        for i in range(n):
            r = eng.open_request(f"b{i}")
            r.input_ids = torch.randint(3, cfg.vocab_size, (length,), generator=g).tolist()
            r.blocks = eng._alloc_blocks(eng._blocks_needed(length + 32))
            reqs.append(r)
        return reqs

    for n, length in prefill:
        reqs = opened(n, length)
        for r in reqs:
            r.chunk = (0, length)
        ev = []
        for i in range(iters + 2):
            # the inputs of a step go to the device before the clock starts: this is the model's own time
            hook = _TimedForward(eng.model)
            eng._forward_pieces(reqs)
            hook.close()
            ev.append(hook)
        torch.cuda.synchronize()
        ms = sorted(h.elapsed() for h in ev[2:])[iters // 2]
        out["prefill"].append({"sequences": n, "length": length, "ms": ms, "tokens_per_s": n * length / ms * 1e3})
        for r in reqs:
            eng.close_request(r.rid)
    for n, ctx_len in decode:
        reqs = opened(n, ctx_len)
        for i in range(0, n, 8):
            for r in reqs[i:i + 8]:
                r.chunk = (0, ctx_len)
            eng._forward_pieces(reqs[i:i + 8])
        run = eng.runner
        for r in reqs:
            run.attach(r)
        run._set_rows(reqs)
        run.d_i32.copy_(run.h_i32)
        run.d_i64.copy_(run.h_i64)
        key = (run._bucket(run.high), False)
        run._capture(key)
        for _ in range(3):
            run.graphs[key].replay()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(20):
            run.graphs[key].replay()
        e1.record()
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1) / 20
        out["decode"].append({"rows": n, "context": ctx_len, "ms": ms, "tokens_per_s": n / ms * 1e3, "launches": run.launches_per_graph[key]})
        for r in reqs:
            eng.close_request(r.rid)
        run.reset_graphs()
    return out


class _TimedForward:
    """CUDA events around one call of a model's forward."""

    def __init__(self, model):
        self.e0, self.e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        self.h = [model.register_forward_pre_hook(lambda *_: self.e0.record()), model.register_forward_hook(lambda *_: self.e1.record())]

    def close(self):
        for h in self.h:
            h.remove()

    def elapsed(self) -> float:
        return self.e0.elapsed_time(self.e1)


def _ragged(lens, bs: int = 64):
    """A batch of (first position, new tokens) pieces on a fresh block table (device tensors), and the blocks it needs."""
    from ..models.qwen3 import SHORT_Q, ForwardMeta, RaggedBatch

    pos, slots, seq, cu, nb = [], [], [], [0], 0
    bt = torch.zeros(len(lens), max(-(-(s + n) // bs) for s, n in lens), dtype=torch.int32)
    for b, (s, n) in enumerate(lens):
        k = -(-(s + n) // bs)
        bt[b, :k] = torch.arange(nb, nb + k)
        pos += range(s, s + n)
        slots += [(nb + p // bs) * bs + p % bs for p in range(s, s + n)]
        seq += [b] * n
        cu.append(cu[-1] + n)
        nb += k
    n_long = sum(n > SHORT_Q for _, n in lens)
    i32 = dict(dtype=torch.int32, device="cuda")
    return ForwardMeta(
        positions=torch.tensor(pos, **i32), block_table=bt.cuda(), slot_mapping=torch.tensor(slots, device="cuda"),
        state_slots=torch.arange(len(lens), **i32),
        ragged=RaggedBatch(cu_q=torch.tensor(cu, **i32) if n_long else None, token_seq=torch.tensor(seq, **i32) if n_long else None,
                           q_lens=[n for _, n in lens], seq_lens=[s + n for s, n in lens], n_long=n_long, t_long=cu[n_long])), nb


class _Rows:
    """Timed kernels: device time and fraction of the roofline, max(bytes ÷ copy bandwidth, FLOPs ÷ GEMM rate) ÷ time."""

    def __init__(self):
        self.bw, self.fl, self.which = peaks()
        self.tm = _Timer()
        self.rows: list[dict] = []

    def add(self, name, like, shape, fn, nbytes, flops=0.0):
        ms = self.tm.ms(fn)
        ideal = max(nbytes / self.bw, flops / self.fl) * 1e3
        self.rows.append({"kernel": name, "like": like, "shape": shape, "us": round(ms * 1e3, 1), "GB/s": round(nbytes / ms / 1e6),
                          "TFLOP/s": round(flops / ms / 1e9, 1), "of_roofline": round(ideal / ms, 3), "peaks": self.which})


def _randn(*shape, dtype=torch.bfloat16):
    return torch.randn(*shape, device="cuda").to(dtype)


@torch.no_grad()
def latent_kernels(cfg, base) -> list[dict]:
    from ..models.layered import LatentSpec, LinearStateSpec
    from ..ops import cuda as K
    from ..ops import mixers as MX
    from ..ops import mixers_cuda as MC

    out = _Rows()
    add, t, rows = out.add, _randn, out.rows
    D = cfg.hidden_size
    lat = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, LatentSpec))
    lin = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, LinearStateSpec))
    ff = next(s.mlp.ff for s in cfg.layer_specs if s.mlp is not None)
    lay = MX.LatentLayout(lat.heads, lat.dim, lat.rot_dim, lat.vdim, lat.kv_rank)
    sizes = [lay.heads, lay.dim, lay.rot, lay.vdim, lay.rank, lay.rank_p, lay.pitch]
    H, sink, err = lat.heads, t(lat.heads), K.C.error_flag(torch.empty(0, device="cuda"))
    for n, length in ((1, 8192), (8, 1024)):
        T = n * length
        m, nb = _ragged([(0, length)] * n)
        cu_k, _, total, max_q = MC._key_ranges(m, lat.window)
        qn = (lat.dim + 63) // 64 * 64
        q, kv, lt, o = t(T, H, qn + 64), t(total, H * (lat.dim + lat.vdim)), t(total, lay.pitch), t(T, H, lat.vdim)
        w = lat.window or length
        pairs = n * sum(min(i + 1, w) for i in range(length))
        add("latent_prefill (tcgen05, window, sink)", "flash_fwd_tc", f"{n}x{length} window {w}",
            lambda: K.C.latent_prefill(q, kv, lt, o, sink, m.ragged.cu_q, cu_k, n, max_q, lat.scale, lat.window, sizes, err),
            2 * (q.numel() + kv.numel() + total * lat.rot_dim + o.numel()), 2.0 * pairs * H * (lat.dim + lat.rot_dim + lat.vdim))
        hq, hk, d = base.num_heads, base.num_kv_heads, base.head_dim
        q2, k2, v2 = t(T, hq, d), t(T, hk, d), t(T, hk, d)
        cu = m.ragged.cu_q
        add("flash_fwd_tc", "", f"{n}x{length}", lambda: K.attention_varlen(q2, k2, v2, cu, length), 2 * (2 * q2.numel() + 2 * k2.numel()),
            2.0 * n * length * (length + 1) / 2 * hq * 2 * d)
        proj, dec = t(T, lin.heads * 2 * (lin.dim + lin.vdim)), torch.tensor(lin.decay, device="cuda")
        st = torch.zeros(n, lin.heads, lin.dim, lin.vdim, device="cuda")
        C = 64
        add("linear_chunk (segments + scan + outputs)", "flash_fwd_tc", f"{n}x{length}",
            lambda: MC.linear_state(proj, lin.heads, lin.dim, lin.vdim, dec, st, m), 2 * T * lin.heads * (2 * lin.dim + 2 * lin.vdim) + 8 * st.numel(),
            2.0 * T * lin.heads * ((C + 1) / 2 * (lin.dim + lin.vdim) + 2 * lin.dim * lin.vdim))
        del q, kv, lt, o, q2, k2, v2, proj, st
    for B, ctx in ((1, 4096), (8, 4096), (64, 4096)):
        m, nb = _ragged([(ctx - 1, 1)] * B)
        cache = t(nb, 64, lay.pitch)
        qa, ol = t(B, H, lay.pitch), t(B, H, lay.rank)
        w = min(lat.window or ctx, ctx)
        splits = MC.decode_splits(B, H, w, 64)
        po, pm = torch.empty(B * H * splits * lay.rank_p, device="cuda"), torch.empty(B * H * splits * 2, device="cuda")
        add("latent_decode + merge", "paged_decode", f"{B} rows, window {w}",
            lambda: K.C.latent_decode(qa, cache, m.block_table, None, m.positions, m.slot_mapping, sink, po, pm, ol, lat.scale, lat.window, splits, sizes, err),
            2 * B * (w * (lay.rank + lay.rot) + H * (lay.pitch + lay.rank)), 2.0 * B * w * H * (2 * lay.rank + lay.rot))
        kc, vc = t(nb, 64, base.num_kv_heads, base.head_dim), t(nb, 64, base.num_kv_heads, base.head_dim)
        q2 = t(B, base.num_heads, base.head_dim)
        L = torch.full((B,), w, dtype=torch.int32, device="cuda")
        add("paged_decode + merge", "", f"{B} rows, context {w}", lambda: K.paged_attention(q2, kc, vc, m.block_table, L),
            2 * B * (w * 2 * base.num_kv_heads * base.head_dim + 2 * base.num_heads * base.head_dim), 4.0 * B * w * base.num_heads * base.head_dim)
        wu = t(H, lat.dim, lat.kv_rank)
        qn, wv, ov = t(B, H, lat.dim), t(H, lat.vdim, lat.kv_rank), t(B, H, lat.vdim)
        add("head_linear (key up-projection into q)", "gemv", f"{B} rows", lambda: K.C.head_linear_mma(qn, wu, False, qa[..., :lay.rank]),
            2 * (wu.numel() + qn.numel() + B * H * lay.rank), 2.0 * B * wu.numel())
        add("head_linear (value up-projection)", "gemv", f"{B} rows", lambda: K.C.head_linear_mma(ol, wv, True, ov),
            2 * (wv.numel() + ol.numel() + ov.numel()), 2.0 * B * wv.numel())
        wo = torch.nn.Parameter(t(H * lat.vdim, lat.kv_rank))
        xo = t(B, lat.kv_rank)
        add("gemv / gemm of as many weight bytes", "", f"{B} rows", lambda: K.gemm_nt(xo, wo.data), 2 * (wo.numel() + xo.numel() + B * wo.shape[0]),
            2.0 * B * wo.numel())
        proj, dec = t(B, lin.heads * 2 * (lin.dim + lin.vdim)), torch.tensor(lin.decay, device="cuda")
        st = torch.zeros(B, lin.heads, lin.dim, lin.vdim, device="cuda")
        add("linear_state step", "paged_decode", f"{B} rows", lambda: MC.linear_state(proj, lin.heads, lin.dim, lin.vdim, dec, st, m),
            8 * st.numel() + 2 * B * lin.heads * (2 * lin.dim + 2 * lin.vdim))
        del cache, kc, vc, st
    for T in (8, 8192):
        x, y, v = t(T, D, dtype=torch.float32), t(T, D), t(D)
        add("output_norm (fp32 residual)", "add_rmsnorm", f"{T} rows", lambda: MC.output_norm_residual(x, y, v, v, 1e-6), T * D * 12)
        r2 = t(T, D)
        add("add_rmsnorm", "", f"{T} rows", lambda: K.add_rmsnorm(y, r2, v, 1e-6), T * D * 8)
        h = t(T, 2 * ff)
        add("clamped_glu", "swiglu", f"{T} rows", lambda: MC.clamped_glu(h, 7.0, 1.702), 6 * T * ff)
        add("swiglu", "", f"{T} rows", lambda: K.swiglu(h), 6 * T * ff)
        o, gt = t(T, lin.heads * lin.vdim), t(T, lin.heads * lin.vdim)
        gw = t(lin.heads * lin.vdim)
        add("gated_norm", "add_rmsnorm", f"{T} rows", lambda: MC.gated_norm(o, gw, gt, 1e-6), 6 * o.numel())
        m, nb = _ragged([(0, T)] if T > 8 else [(4000, 1)] * T)
        cache = t(nb, 64, lay.pitch)
        proj = t(T, lay.q_rows + lay.rank + lay.rot)
        freq = torch.tensor(lat.rotary.table()[0], dtype=torch.float64, device="cuda")
        kn = t(lay.rank)
        tl = m.ragged.t_long
        qa, qf = t(T - tl, H, lay.pitch), t(tl, H, (lat.dim + 63) // 64 * 64 + 64)
        add("latent_prep (rotate, norm, cache)", "qk_norm_rope_cache", f"{T} rows",
            lambda: K.C.latent_prep(proj, m.positions, m.slot_mapping, freq, 1.0, kn, 1e-6, cache, qa, qf, tl, (lat.dim + 63) // 64 * 64,
                                    (lat.dim + 63) // 64 * 64 + 64, sizes),
            2 * T * (lay.rank + 2 * lay.rot + lay.pitch + H * (lay.rot * 2 if T <= 8 else lay.dim * 2 + lay.rot * 2)))
        q2, k2, v2 = t(T, base.num_heads, base.head_dim), t(T, base.num_kv_heads, base.head_dim), t(T, base.num_kv_heads, base.head_dim)
        qw = t(base.head_dim)
        kc, vc = t(nb, 64, base.num_kv_heads, base.head_dim), t(nb, 64, base.num_kv_heads, base.head_dim)
        add("qk_norm_rope_cache", "", f"{T} rows", lambda: K.qk_norm_rope_cache(q2, k2, v2, qw, qw, m.positions, 1e6, 1e-6, kc, vc, m.slot_mapping),
            2 * (2 * q2.numel() + 5 * k2.numel()))
    return rows


@torch.no_grad()
def attention_kernels(cfg, base) -> list[dict]:
    """Windowed grouped-query attention, routed clamped experts and the fused sums beside the grouped-query mixture's kernels."""
    from dataclasses import replace

    from ..ops import cuda as K
    from ..ops import mixers as MX
    from ..ops import mixers_cuda as MC

    out = _Rows()
    add, t = out.add, _randn
    spec = cfg.layer_specs[0]
    m, f, D = spec.mixer, spec.mlp, cfg.hidden_size
    lay = MX.AttentionLayout(m.heads, m.kv_heads, m.dim, m.vdim, m.rotary.dims, m.window, m.keep_first)
    hq, hk, d = base.num_heads, base.num_kv_heads, base.head_dim
    H, G, err, sink = m.heads, m.kv_heads, K.C.error_flag(torch.empty(0, device="cuda")), t(m.heads)

    def sizes(l):
        return [l.heads, l.kv_heads, l.dim, l.vdim, l.rot, l.window, l.keep, -(-l.dim // 64) * 64]

    for n, length in ((1, 8192), (8, 1024), (1, 1024)):
        T = n * length
        meta, nb = _ragged([(0, length)] * n)
        q, kc, vc, o = t(T, H, -(-m.dim // 64) * 64), t(nb, 64, G, m.dim), t(nb, 64, G, m.vdim), t(T, H * m.vdim)
        for l in (lay, replace(lay, window=0, keep=0)):
            if l.window >= length:
                continue
            pairs = n * sum(min(i + 1, l.window + min(l.keep, max(0, i + 1 - l.window))) if l.window else i + 1 for i in range(length))
            add("window_prefill (tcgen05, pages, sink)", "flash_fwd_tc", f"{n}x{length} window {l.window} + {l.keep}",
                lambda: K.C.window_prefill(q, kc, vc, o, sink, meta.ragged.cu_q, meta.positions, meta.block_table, n, length, T, m.scale, sizes(l), err),
                2 * (q.numel() + kc.numel() + vc.numel() + o.numel()), 2.0 * pairs * H * (m.dim + m.vdim))
        q2, k2, v2 = t(T, hq, d), t(T, hk, d), t(T, hk, d)
        add("flash_fwd_tc", "", f"{n}x{length}", lambda: K.attention_varlen(q2, k2, v2, meta.ragged.cu_q, length), 2 * (2 * q2.numel() + 2 * k2.numel()),
            2.0 * n * length * (length + 1) / 2 * hq * 2 * d)
    del q, kc, vc, o, q2, k2, v2
    for B, ctx in ((1, 4096), (8, 4096), (64, 4096)):
        meta, nb = _ragged([(ctx - 1, 1)] * B)
        kc, vc, o = t(nb, 64, G, m.dim), t(nb, 64, G, m.vdim), t(B, H * m.vdim)
        q = t(B, H, -(-m.dim // 64) * 64)
        n_keys = m.window + m.keep_first
        add("window_decode (cluster splits, sink)", "paged_decode", f"{B} rows, {n_keys} keys",
            lambda: K.C.window_decode(q, kc, vc, meta.block_table, None, meta.positions, meta.slot_mapping, sink, o, m.scale,
                                      MC.window_splits(B, lay), sizes(lay)),
            2 * B * (n_keys * G * (m.dim + m.vdim) + H * (m.dim + m.vdim)), 2.0 * B * n_keys * H * (m.dim + m.vdim))
        kb, vb, q2 = t(nb, 64, hk, d), t(nb, 64, hk, d), t(B, hq, d)
        L = torch.full((B,), n_keys, dtype=torch.int32, device="cuda")
        add("paged_decode + merge", "", f"{B} rows, {n_keys} keys", lambda: K.paged_attention(q2, kb, vb, meta.block_table, L),
            2 * B * (n_keys * 2 * hk * d + 2 * hq * d), 4.0 * B * n_keys * hq * d)
        del kc, vc, kb, vb
    freq = torch.tensor(m.rotary.table()[0], dtype=torch.float64, device="cuda")
    qn, kn, nw, w_in = t(H * m.dim), t(G * m.dim), t(D), torch.nn.Parameter(t(lay.rows + 2 * f.shared.ff, D))
    router, bias, w_out = torch.nn.Parameter(t(f.experts, D)), t(f.experts), torch.nn.Parameter(t(D, H * m.vdim + f.shared.ff))
    wqkv, wo = torch.nn.Parameter(t(base.qkv_size, D)), torch.nn.Parameter(t(D, base.q_size))
    for T in (8, 8192):
        meta, nb = _ragged([(0, T)] if T > 8 else [(4000, 1)] * T)
        kc, vc = t(nb, 64, G, m.dim), t(nb, 64, G, m.vdim)
        proj, q, both = t(T, w_in.shape[0]), t(T, H, -(-m.dim // 64) * 64), t(T, w_out.shape[1])
        logits, w, idx = t(T, f.experts, dtype=torch.float32), torch.empty(T, f.top, device="cuda"), torch.empty(T, f.top, dtype=torch.int32, device="cuda")
        add("window_prep (norm, rotate, cache, experts, glu)", "qk_norm_rope_cache", f"{T} rows",
            lambda: K.C.window_prep(proj, meta.positions, meta.slot_mapping, freq, 1.0, qn, kn, 1e-6, kc, vc, q, sizes(lay),
                                    [logits, w, idx, proj[:, lay.rows:], both[:, H * m.vdim:], None], [7.0, 1.702, 1.0, 1.0], [0, 1, 1]),
            2 * T * (2 * lay.rows + 3 * f.shared.ff) + 4 * T * f.experts)
        q2, k2, v2, qw = t(T, hq, d), t(T, hk, d), t(T, hk, d), t(d)
        kb, vb = t(nb, 64, hk, d), t(nb, 64, hk, d)
        add("qk_norm_rope_cache", "", f"{T} rows", lambda: K.qk_norm_rope_cache(q2, k2, v2, qw, qw, meta.positions, 1e6, 1e-6, kb, vb, meta.slot_mapping),
            2 * (2 * q2.numel() + 5 * k2.numel()))
        add("router_topk", "", f"{T} rows", lambda: K.router_topk(logits, f.top), 4 * T * f.experts)
        x, to, y, r2 = t(T, D, dtype=torch.float32), t(T, D, dtype=torch.float32), t(T, D), t(T, D)
        add("sum_norm (fp32 residual, one addend)", "add_rmsnorm", f"{T} rows", lambda: MC.sum_norm(x, to, [MX.Addend(y)], None, nw, 1e-6), T * D * 12)
        add("add_rmsnorm", "", f"{T} rows", lambda: K.add_rmsnorm(y, r2, nw, 1e-6), T * D * 8)
        if T > 8:
            bt = 128
            xp, seg, tile, dst = K.sort_by_expert(y, torch.rand(T, f.experts, device="cuda").topk(f.top).indices.int(), f.experts, bt)
            a = MX.Addend(t(*xp.shape), w.uniform_(), dst)
            add("sum_norm (one addend, experts' rows)", "moe_combine + add_rmsnorm", f"{T} rows",
                lambda: MC.sum_norm(x, to, [MX.Addend(y), a], None, nw, 1e-6), T * D * (12 + 2 * f.top))
            add("moe_combine + add_rmsnorm", "", f"{T} rows",
                lambda: (K.C.moe_combine(a.y, a.weights, dst, r2, f.top), K.add_rmsnorm(y, r2, nw, 1e-6)), T * D * (2 * f.top + 2 + 8))
    for T in (1, 4):
        x, y, y2, r2 = t(T, D, dtype=torch.float32), t(T, D), t(T, D), t(T, D)
        add("sum_norm_linear (+ router)", "add_rmsnorm_linear", f"{T} rows",
            lambda: MC.sum_norm_linear(x, [MX.Addend(y), MX.Addend(y2)], None, nw, 1e-6, w_in, router, bias, True),
            2 * (w_in.numel() + router.numel()))
        add("add_rmsnorm_linear", "", f"{T} rows", lambda: K.add_rmsnorm_linear(y, r2, nw, 1e-6, wqkv), 2 * wqkv.numel())
    for T in (1, 8, 64, 8192):
        h = t(T, D)
        w13, w2 = t(f.experts, 2 * f.expert.ff, D), t(f.experts, D, f.expert.ff)
        idx = torch.rand(T, f.experts, device="cuda").topk(f.top).indices.int()
        w = torch.rand(T, f.top, device="cuda")
        used = idx.unique().numel()
        nbytes, flops = 2.0 * used * 3 * D * f.expert.ff + 4 * T * D, 6.0 * T * f.top * D * f.expert.ff
        add("routed_experts (clamped; sum left to sum_norm)" if T > 8 else "routed_experts (clamped)", "moe_ffn", f"{T} rows, {used} experts",
            lambda: MC.routed_experts(h, w13, w2, w, idx, f.expert.limit, f.expert.alpha), nbytes, flops)
        add("moe_ffn", "", f"{T} rows, {used} experts", lambda: K.moe_ffn(h, w13, w2, w, idx), nbytes, flops)
        both = t(T, w_out.shape[1])
        add("output projection (heads and shared expert)", "wo", f"{T} rows", lambda: K.linear(both, w_out), 2.0 * (w_out.numel() + both.numel() + T * D),
            2.0 * T * w_out.numel())
        ob = t(T, wo.shape[1])
        add("wo", "", f"{T} rows", lambda: K.linear(ob, wo), 2.0 * (wo.numel() + ob.numel() + T * D), 2.0 * T * wo.numel())
    return out.rows


@torch.no_grad()
def hybrid_kernels(cfg, base) -> list[dict]:
    """Differential attention, the state-space mixer, ungated experts and the sums with two norms beside the grouped-query mixture's kernels
    (and beside linear attention with as large a state)."""
    from ..models.layered import DifferentialSpec, MoeSpec, SsmSpec
    from ..ops import cuda as K
    from ..ops import mixers as MX
    from ..ops import mixers_cuda as MC

    out = _Rows()
    add, t = out.add, _randn
    D = cfg.hidden_size
    m = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, DifferentialSpec))
    c = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, SsmSpec))
    f = next(s.mlp for s in cfg.layer_specs if isinstance(s.mlp, MoeSpec))
    lay, ss = MX.DifferentialLayout(m.heads, m.kv_heads, m.dim, m.vdim), MX.SsmLayout(c.heads, c.vdim, c.state, c.groups, c.conv)
    pair, H, G = lay.paired, m.heads, m.kv_heads
    hq, hk, d = base.num_heads, base.num_kv_heads, base.head_dim
    pitch = -(-pair.dim // 64) * 64
    sizes = [pair.heads, pair.kv_heads, pair.dim, pair.vdim, 0, 0, 0, pitch]
    lam, qn, lvec = torch.full((1,), 0.6, device="cuda"), t(m.dim), t(4, m.dim)

    def diff(gates):
        return lam, gates, 0.2, 1e-6

    conv, conv_b, vec, Dv = t(ss.channels, c.conv), t(ss.channels), t(c.heads), t(c.heads)
    lin_h, lin_d = c.heads * c.vdim // c.state, c.state              # linear attention with a state of the same size
    for n, length in ((1, 8192), (8, 1024), (1, 1024)):
        T = n * length
        meta, nb = _ragged([(0, length)] * n)
        q, kc, vc, o, gates = t(T, 2 * H, pitch), t(nb, 64, G, pair.dim), t(nb, 64, G, m.vdim), t(T, H * m.vdim), t(T, H)
        pairs = n * length * (length + 1) / 2
        add("differential prefill (two maps, norm, gate)", "flash_fwd_tc", f"{n}x{length}",
            lambda: MC._paged_attention(q, pair, kc, vc, meta, o, m.scale, None, sizes, True, diff(gates)),
            2 * (T * 2 * H * m.dim + kc.numel() + vc.numel() + o.numel()), 4.0 * pairs * H * (m.dim + m.vdim))
        q2, k2, v2 = t(T, hq, d), t(T, hk, d), t(T, hk, d)
        add("flash_fwd_tc", "", f"{n}x{length}", lambda: K.attention_varlen(q2, k2, v2, meta.ragged.cu_q, length), 2 * (2 * q2.numel() + 2 * k2.numel()),
            4.0 * pairs * hq * d)
        del q, kc, vc, o, q2, k2, v2
        proj, xbc = t(T, ss.inner + ss.channels + c.heads), t(T, ss.channels)
        step, decay = torch.rand(T, c.heads, device="cuda") * 0.1, -torch.rand(T, c.heads, device="cuda") * 0.1
        state, ring = torch.zeros(n, c.heads, c.state, c.vdim, device="cuda"), torch.zeros(n, c.conv, ss.channels, device="cuda")
        w = [conv, conv_b, vec, vec, Dv, state, ring, meta.state_slots, meta.positions]
        segs, seq_segs, multi = MC._segments(meta, c.heads // K.C.ssm_heads_per_cta(c.heads, c.vdim, c.groups))
        seg_state = torch.empty(segs.shape[0], c.heads, c.state, c.vdim, device="cuda") if multi else None
        seg_decay = torch.empty(segs.shape[0], c.heads, device="cuda") if multi else None
        y, S, C = t(T, ss.inner), [c.heads, c.vdim, c.state, c.groups, c.conv], 64
        add("ssm_chunk (segments + scan + outputs, gate)", "linear_chunk", f"{n}x{length}",
            lambda: K.C.ssm_chunk(proj, xbc, step, decay, S, w, segs, seq_segs, seg_state, seg_decay, y),
            2 * T * (2 * ss.inner + ss.channels) + 8 * T * c.heads + 8 * state.numel(),
            2.0 * T * ((C + 1) / 2 * (c.groups * c.state + c.heads * c.vdim) + 2 * c.heads * c.state * c.vdim))
        lin = t(T, lin_h * 4 * lin_d)
        dec, lst = torch.rand(lin_h, device="cuda"), torch.zeros(n, lin_h, lin_d, lin_d, device="cuda")
        add("linear_chunk (segments + scan + outputs)", "", f"{n}x{length}", lambda: MC.linear_state(lin, lin_h, lin_d, lin_d, dec, lst, meta),
            2 * T * lin_h * 4 * lin_d + 8 * lst.numel(), 2.0 * T * lin_h * ((C + 1) / 2 * 2 * lin_d + 2 * lin_d * lin_d))
        tiles = MC._conv_tiles(meta, c.conv)
        add("ssm_conv (convolution, step sizes)", "swiglu", f"{n}x{length}",
            lambda: K.C.ssm_conv(proj, S, w, tiles, meta.ragged.cu_q, xbc, step, decay, *MC._aside(None, T)), 4 * T * ss.channels + 10 * T * c.heads)
        h = t(T, 2 * ss.channels)
        add("swiglu", "", f"{n}x{length}", lambda: K.swiglu(h), 6 * T * ss.channels)
        del proj, xbc, lin, h
    for B, ctx in ((1, 4096), (8, 4096), (64, 4096)):
        meta, nb = _ragged([(ctx - 1, 1)] * B)
        kc, vc, o, gates, q = t(nb, 64, G, pair.dim), t(nb, 64, G, m.vdim), t(B, H * m.vdim), t(B, H), t(B, 2 * H, pitch)
        add("differential decode (two maps, norm, gate)", "paged_decode", f"{B} rows, {ctx} keys",
            lambda: MC._paged_attention(q, pair, kc, vc, meta, o, m.scale, None, sizes, True, diff(gates)),
            2 * B * (ctx * G * (pair.dim + m.vdim) + H * (2 * m.dim + m.vdim)), 4.0 * B * ctx * H * (m.dim + m.vdim))
        kb, vb, q2 = t(nb, 64, hk, d), t(nb, 64, hk, d), t(B, hq, d)
        L = torch.full((B,), ctx, dtype=torch.int32, device="cuda")
        add("paged_decode + merge", "", f"{B} rows, {ctx} keys", lambda: K.paged_attention(q2, kb, vb, meta.block_table, L),
            2 * B * (ctx * 2 * hk * d + 2 * hq * d), 4.0 * B * ctx * hq * d)
        del kc, vc, kb, vb
        proj, y = t(B, ss.inner + ss.channels + c.heads), t(B, ss.inner)
        state, ring = torch.zeros(B, c.heads, c.state, c.vdim, device="cuda"), torch.zeros(B, c.conv, ss.channels, device="cuda")
        w = [conv, conv_b, vec, vec, Dv, state, ring, meta.state_slots, meta.positions]
        S = [c.heads, c.vdim, c.state, c.groups, c.conv]
        add("ssm_step (convolution, state, gate)", "linear_state step", f"{B} rows", lambda: K.C.ssm_step(proj, S, w, y, *MC._aside(None, B)),
            8 * state.numel() + 4 * ring.numel() + 2 * B * (2 * ss.inner + ss.channels))
        lin, dec = t(B, lin_h * 4 * lin_d), torch.rand(lin_h, device="cuda")
        lst = torch.zeros(B, lin_h, lin_d, lin_d, device="cuda")
        add("linear_state step", "", f"{B} rows", lambda: MC.linear_state(lin, lin_h, lin_d, lin_d, dec, lst, meta), 8 * lst.numel() + 2 * B * lin_h * 4 * lin_d)
    nw, corr, z = t(D), t(f.experts), t(ss.inner)
    w_in = torch.nn.Parameter(t(ss.inner + ss.channels + c.heads, D))
    router, wo = torch.nn.Parameter(t(f.experts, D)), torch.nn.Parameter(t(D, ss.inner))
    wqkv = torch.nn.Parameter(t(base.qkv_size, D))
    for T in (8, 8192):
        meta, nb = _ragged([(0, T)] if T > 8 else [(4000, 1)] * T)
        kc, vc, q = t(nb, 64, G, pair.dim), t(nb, 64, G, m.vdim), t(T, 2 * H, pitch)
        proj, logits = t(T, lay.gate_at + H), t(T, f.experts, dtype=torch.float32)
        a = MX.Aside(logits=logits, top=f.top, routing=f.routing, correction=corr)
        add("diff_prep (norms, temperature, cache, experts)", "qk_norm_rope_cache", f"{T} rows",
            lambda: K.C.diff_prep(proj, meta.positions, meta.slot_mapping, qn, qn, lvec, lam, kc, vc, q, [H, G, m.dim, m.vdim, pitch], 1e-6, 0.1, 8192.0,
                                  0.8, *MC._aside(a, T)),
            2 * T * (2 * lay.gate_at + 2 * H * m.dim) + 4 * T * f.experts)
        q2, k2, v2, qw = t(T, hq, d), t(T, hk, d), t(T, hk, d), t(d)
        kb, vb = t(nb, 64, hk, d), t(nb, 64, hk, d)
        add("qk_norm_rope_cache", "", f"{T} rows", lambda: K.qk_norm_rope_cache(q2, k2, v2, qw, qw, meta.positions, 1e6, 1e-6, kb, vb, meta.slot_mapping),
            2 * (2 * q2.numel() + 5 * k2.numel()))
        add("router_topk", "", f"{T} rows", lambda: K.router_topk(logits, f.top), 4 * T * f.experts)
        y, y2 = t(T, ss.inner), t(T, ss.inner)
        add("part_norm (state-space output)", "add_rmsnorm", f"{T} rows", lambda: K.C.part_norm(y, z, y2, c.norm_groups, 1e-6), 4 * y.numel())
        x, to, o, r2 = t(T, D, dtype=torch.float32), t(T, D, dtype=torch.float32), t(T, D), t(T, D)
        add("sum_norm (one scaled addend, two norms)", "add_rmsnorm", f"{T} rows",
            lambda: MC.sum_norm(x, to, [MX.Addend(o, scale=nw)], None, nw, 1e-6, 1.0, 1.0, nw), T * D * 14)
        add("add_rmsnorm", "", f"{T} rows", lambda: K.add_rmsnorm(o, r2, nw, 1e-6), T * D * 8)
        if T > 8:
            xp, seg, tile, dst = K.sort_by_expert(o, torch.rand(T, f.experts, device="cuda").topk(f.top).indices.int(), f.experts, 128)
            e = MX.Addend(t(*xp.shape), torch.rand(T, f.top, device="cuda"), dst, nw)
            add("sum_norm (addend, experts' rows, two norms)", "moe_combine + add_rmsnorm", f"{T} rows",
                lambda: MC.sum_norm(x, to, [MX.Addend(o, scale=nw), e], None, nw, 1e-6, 1.0, 1.0, nw), T * D * (14 + 2 * f.top))
            add("moe_combine + add_rmsnorm", "", f"{T} rows",
                lambda: (K.C.moe_combine(e.y, e.weights, dst, r2, f.top), K.add_rmsnorm(o, r2, nw, 1e-6)), T * D * (2 * f.top + 2 + 8))
    for T in (1, 4):
        x, o, o2, r2 = t(T, D, dtype=torch.float32), t(T, D), t(T, D), t(T, D)
        add("sum_two_norms_linear (+ router)", "add_rmsnorm_linear", f"{T} rows",
            lambda: MC.sum_two_norms_linear(x, [MX.Addend(o, scale=nw), MX.Addend(o2, scale=nw)], nw, w_in, nw, router, 1e-6, 1.0, True),
            2 * (w_in.numel() + router.numel()))
        add("add_rmsnorm_linear", "", f"{T} rows", lambda: K.add_rmsnorm_linear(o, r2, nw, 1e-6, wqkv), 2 * wqkv.numel())
        y = t(T, ss.inner)
        add("part_norm_linear (norm inside the output projection)", "add_rmsnorm_linear", f"{T} rows",
            lambda: MC.part_norm_linear(y, z, c.norm_groups, 1e-6, wo), 2 * wo.numel())
    for T in (1, 8, 64, 8192):
        h = t(T, D)
        w1, w2 = t(f.experts, f.up_rows, D), t(f.experts, D, f.expert.ff)
        Fb = base.moe_ffn_hidden_size
        b13, b2 = t(f.experts, 2 * Fb, D), t(f.experts, D, Fb)
        idx = torch.rand(T, f.experts, device="cuda").topk(f.top).indices.int()
        w = torch.rand(T, f.top, device="cuda")
        used = idx.unique().numel()
        nbytes, flops = 2.0 * used * 2 * D * f.expert.ff + 4 * T * D, 4.0 * T * f.top * D * f.expert.ff
        add("routed_experts (squared relu; sum left to sum_norm)" if T > 8 else "routed_experts (squared relu)", "moe_ffn", f"{T} rows, {used} experts",
            lambda: MC.routed_experts(h, w1, w2, w, idx, 0.0, 0.0, 0.0, True), nbytes, flops)
        add("moe_ffn", "", f"{T} rows, {used} experts", lambda: K.moe_ffn(h, b13, b2, w, idx), 2.0 * used * 3 * D * Fb + 4 * T * D, 6.0 * T * f.top * D * Fb)
    return out.rows


@torch.no_grad()
def delta_kernels(cfg, base) -> list[dict]:
    """Gated delta rule, chunked attention with a distance bias, gated latent attention and the pre-norm arrangement's row-wise kernels beside
    those of a model with latent and linear attention (`base`)."""
    from ..models.layered import AttentionSpec, DeltaSpec, LatentSpec, LinearStateSpec
    from ..ops import cuda as K
    from ..ops import mixers as MX
    from ..ops import mixers_cuda as MC

    out = _Rows()
    add, t = out.add, _randn
    D, ff = cfg.hidden_size, next(s.mlp.ff for s in cfg.layer_specs if s.mlp is not None)

    def first(c, kind):
        return next(s.mixer for s in c.layer_specs if isinstance(s.mixer, kind))

    m, a, l, lin, wl = first(cfg, DeltaSpec), first(cfg, AttentionSpec), first(cfg, LatentSpec), first(base, LinearStateSpec), first(base, LatentSpec)
    ds = MX.DeltaLayout(m.heads, m.kv_heads, m.dim, m.vdim, m.conv, m.decay_rank, m.gate_rank)
    al = MX.AttentionLayout(a.heads, a.kv_heads, a.dim, a.vdim, 0, 0, 0, a.chunk, True, True)
    pitch = -(-a.dim // 64) * 64
    asz = [a.heads, a.kv_heads, a.dim, a.vdim, 0, 0, 0, pitch, a.chunk]
    H, G, err = a.heads, a.kv_heads, K.C.error_flag(torch.empty(0, device="cuda"))
    r1, r2, sink = torch.rand(H, device="cuda").bfloat16(), torch.rand(H, device="cuda").bfloat16(), t(wl.heads)

    def latent_sizes(s):
        y = MX.LatentLayout(s.heads, s.dim, s.rot_dim, s.vdim, s.kv_rank)
        return y, [y.heads, y.dim, y.rot, y.vdim, y.rank, y.rank_p, y.pitch]

    conv, A, dtb, nv = t(ds.channels, m.conv), t(m.heads) - 2, t(m.heads * m.dim) - 2, t(m.vdim)
    S = [m.heads, m.kv_heads, m.dim, m.vdim, m.conv, ds.beta_at]
    n_state = m.heads * m.dim * m.vdim
    for n, length in ((1, 8192), (8, 1024), (1, 1024)):
        T, shape = n * length, f"{n}x{length}"
        meta, nb = _ragged([(0, length)] * n)
        proj, act, raw, gate, y = t(T, ds.beta_at + m.heads), t(T, ds.channels), t(T, m.heads * m.dim), t(T, m.heads * m.vdim), t(T, m.heads * m.vdim)
        state, ring = torch.zeros(n, m.heads, m.dim, m.vdim, device="cuda"), torch.zeros(n, m.conv, ds.channels, device="cuda")
        w = [conv, A, dtb, state, ring, meta.state_slots, meta.positions, raw]
        rounds = MC._chunk_rounds(meta, ds)
        scratch = torch.empty(max(c.shape[0] for c, _ in rounds) * m.heads * K.C.delta_chunk_bytes(m.dim, m.vdim), dtype=torch.uint8, device="cuda")

        def chunks():
            for c, p in rounds:
                K.C.delta_chunk(proj, act, S, w, c, p, scratch, MC.scan_warps(p.shape[0] * m.heads, m.vdim), y, err)

        C = 64
        # the mathematics in chunks: two triangles of key products, the triangular solve on values and keys, three products with the state
        flops = 2.0 * T * m.heads * ((C + 1) / 2 * (2 * m.dim + (m.dim + m.vdim) + m.vdim) + 3 * m.dim * m.vdim)
        add("delta_chunk (decays, triangles, scan)", "linear_chunk", shape, chunks, 2 * T * (ds.channels + m.heads * (m.dim + 1 + m.vdim)) + 8 * state.numel(), flops)
        lp, dec = t(T, lin.heads * 2 * (lin.dim + lin.vdim)), torch.tensor(lin.decay, device="cuda")
        ls = torch.zeros(n, lin.heads, lin.dim, lin.vdim, device="cuda")
        add("linear_chunk (segments + scan + outputs)", "", shape, lambda: MC.linear_state(lp, lin.heads, lin.dim, lin.vdim, dec, ls, meta),
            2 * T * lin.heads * (2 * lin.dim + 2 * lin.vdim) + 8 * ls.numel(), 2.0 * T * lin.heads * ((C + 1) / 2 * (lin.dim + lin.vdim) + 2 * lin.dim * lin.vdim))
        tiles = MC._conv_tiles(meta, m.conv)
        add("delta_conv", "swiglu", shape, lambda: K.C.delta_conv(proj, S, w, tiles, meta.ragged.cu_q, act), 4 * T * ds.channels)
        h = t(T, 2 * ds.channels)
        add("swiglu", "", shape, lambda: K.swiglu(h), 6 * T * ds.channels)
        g2 = torch.empty_like(y)
        add("head_gated_norm", "gated_norm", shape, lambda: K.C.head_gated_norm(y, nv, gate, g2, 1e-6), 6 * y.numel())
        gw = t(m.heads * m.vdim)
        add("gated_norm", "", shape, lambda: K.C.gated_norm(y, gw, gate, g2, 1e-6), 6 * y.numel())
        del proj, act, raw, scratch, lp, h
        q, kc, vc, o, og = t(T, H, pitch), t(nb, 64, G, a.dim), t(nb, 64, G, a.vdim), t(T, H * a.vdim), t(T, H * a.vdim)
        pairs = n * sum(i % a.chunk + 1 for i in range(length))
        add(f"window_prefill (chunks of {a.chunk}, distance bias, gate)", "flash_fwd_tc", shape,
            lambda: K.C.window_prefill(q, kc, vc, o, None, meta.ragged.cu_q, meta.positions, meta.block_table, n, length, T, a.scale, asz, err, r1=r1, r2=r2, out_gate=og),
            2 * (q.numel() + kc.numel() + vc.numel() + 2 * o.numel()), 2.0 * pairs * H * (a.dim + a.vdim))
        q2, k2, v2 = t(T, H, a.dim), t(T, G, a.dim), t(T, G, a.vdim)
        add("flash_fwd_tc", "", shape, lambda: K.attention_varlen(q2, k2, v2, meta.ragged.cu_q, length), 2 * (2 * q2.numel() + 2 * k2.numel()),
            2.0 * n * length * (length + 1) / 2 * H * 2 * a.dim)
        del q, kc, vc, o, og, q2, k2, v2
        for name, s, like in (("latent_prefill (all keys, gate)", l, "latent_prefill of the other model"), ("latent_prefill of the other model (window, sink)", wl, "")):
            y_, sz = latent_sizes(s)
            cu_k, _, total, max_q = MC._key_ranges(meta, s.window)
            q, kv, lt, o, og = t(T, s.heads, (s.dim + 63) // 64 * 64 + 64), t(total, s.heads * (s.dim + s.vdim)), t(total, y_.pitch), t(T, s.heads, s.vdim), t(T, s.heads * s.vdim)
            wn = s.window or length
            pairs = n * sum(min(i + 1, wn) for i in range(length))
            add(name, like, shape, lambda: K.C.latent_prefill(q, kv, lt, o, sink if s.sink else None, meta.ragged.cu_q, cu_k, n, max_q, s.scale, s.window, sz, err,
                                                              og if s.gate else None),
                2 * (q.numel() + kv.numel() + total * s.rot_dim + o.numel() * (2 if s.gate else 1)), 2.0 * pairs * s.heads * (s.dim + s.rot_dim + s.vdim))
            del q, kv, lt, o, og
    for B, ctx in ((1, 4096), (8, 4096), (64, 4096)):
        shape = f"{B} rows"
        meta, nb = _ragged([(ctx - 1, 1)] * B)
        proj, raw, gate, y = t(B, ds.beta_at + m.heads), t(B, m.heads * m.dim), t(B, m.heads * m.vdim), t(B, m.heads * m.vdim)
        state, ring = torch.zeros(B, m.heads, m.dim, m.vdim, device="cuda"), torch.zeros(B, m.conv, ds.channels, device="cuda")
        w = [conv, A, dtb, state, ring, meta.state_slots, meta.positions, raw]
        add("delta_step (convolution, state, gated norm)", "linear_state step", shape, lambda: K.C.delta_step(proj, S, w, nv, gate, 1e-6, y),
            8 * state.numel() + 4 * ring.numel() + 2 * B * (ds.channels + m.heads * (m.dim + 2 * m.vdim)))
        lp, dec = t(B, lin.heads * 2 * (lin.dim + lin.vdim)), torch.tensor(lin.decay, device="cuda")
        ls = torch.zeros(B, lin.heads, lin.dim, lin.vdim, device="cuda")
        add("linear_state step", "", shape, lambda: MC.linear_state(lp, lin.heads, lin.dim, lin.vdim, dec, ls, meta), 8 * ls.numel() + 2 * B * lin.heads * 2 * (lin.dim + lin.vdim))
        del state, ring, ls
        q, kc, vc, o, og = t(B, H, pitch), t(nb, 64, G, a.dim), t(nb, 64, G, a.vdim), t(B, H * a.vdim), t(B, H * a.vdim)
        keys = (ctx - 1) % a.chunk + 1
        add("window_decode (chunk, distance bias, gate)", "paged_decode", f"{shape}, {keys} keys",
            lambda: K.C.window_decode(q, kc, vc, meta.block_table, None, meta.positions, meta.slot_mapping, None, o, a.scale, MC.window_splits(B, al), asz, r1=r1,
                                      r2=r2, out_gate=og), 2 * B * (keys * G * (a.dim + a.vdim) + H * (a.dim + 2 * a.vdim)), 2.0 * B * keys * H * (a.dim + a.vdim))
        L, q2 = torch.full((B,), keys, dtype=torch.int32, device="cuda"), t(B, H, a.dim)
        add("paged_decode + merge", "", f"{shape}, {keys} keys", lambda: K.paged_attention(q2, kc, vc, meta.block_table, L),
            2 * B * (keys * G * (a.dim + a.vdim) + H * (a.dim + a.vdim)), 2.0 * B * keys * H * (a.dim + a.vdim))
        del kc, vc
        for name, s, like in (("latent_decode + merge (all keys)", l, "latent_decode of the other model"), ("latent_decode of the other model (window, sink) + merge", wl, "")):
            y_, sz = latent_sizes(s)
            cache, qa, ol = t(nb, 64, y_.pitch), t(B, s.heads, y_.pitch), t(B, s.heads, y_.rank)
            wn = min(s.window or ctx, ctx)
            splits = MC.decode_splits(B, s.heads, s.window, 64)
            po, pm = torch.empty(B * s.heads * splits * y_.rank_p, device="cuda"), torch.empty(B * s.heads * splits * 2, device="cuda")
            add(name, like, f"{shape}, {wn} keys",
                lambda: K.C.latent_decode(qa, cache, meta.block_table, None, meta.positions, meta.slot_mapping, sink if s.sink else None, po, pm, ol, s.scale, s.window,
                                          splits, sz, err),
                2 * B * (wn * (y_.rank + y_.rot) + s.heads * (y_.pitch + y_.rank)), 2.0 * B * wn * s.heads * (2 * y_.rank + y_.rot))
            del cache
        wv, ov, gv = t(l.heads, l.vdim, l.kv_rank), t(B, l.heads, l.vdim), t(B, l.heads * l.vdim)
        add("head_linear (value up-projection, gate)", "head_linear", shape, lambda: K.C.head_linear_mma(ol, wv, True, ov, gv), 2 * (wv.numel() + ol.numel() + 2 * ov.numel()))
        add("head_linear", "", shape, lambda: K.C.head_linear_mma(ol, wv, True, ov), 2 * (wv.numel() + ol.numel() + ov.numel()))
    side, nw = cfg.token_side, t(D)
    table = t(4096, cfg.num_layers * side)
    for T in (8, 8192):
        shape = f"{T} rows"
        meta, nb = _ragged([(0, T)] if T > 8 else [(4000, 1)] * T)
        x, y, r2_ = t(T, D, dtype=torch.float32), t(T, D), t(T, D)
        add("residual_norm (factor, next norm)", "add_rmsnorm", shape, lambda: MC.residual_norm(x, y, None, 0.4, nw, 1e-6, torch.bfloat16), T * D * 12)
        add("residual_norm (normed addend, next norm)", "add_rmsnorm", shape, lambda: MC.residual_norm(x, y, nw, 0.4, nw, 1e-6, torch.bfloat16), T * D * 12)
        add("residual_norm (copy for the token input)", "add_rmsnorm", shape, lambda: MC.residual_norm(x, y, None, 0.4, None, 1e-6, torch.bfloat16), T * D * 12)
        add("add_rmsnorm", "", shape, lambda: K.add_rmsnorm(y, r2_, nw, 1e-6), T * D * 8)
        h, act2 = t(T, ff), t(2)
        add("xielu", "swiglu", shape, lambda: MC.xielu(h, act2), 4 * T * ff)
        h2 = t(T, 2 * ff)
        add("swiglu", "", shape, lambda: K.swiglu(h2), 6 * T * ff)
        z, tok = t(T, side), torch.randint(0, 4096, (T,), dtype=torch.int32, device="cuda")
        add("gelu_rows", "swiglu", shape, lambda: MC.gelu_times_rows(z, tok, table, side), 6 * T * side)
        h3 = t(T, 2 * side)
        add("swiglu", "", f"{shape} of {side}", lambda: K.swiglu(h3), 6 * T * side)
        proj, q = t(T, al.rows + H * a.vdim), t(T, H, pitch)
        kc, vc = t(nb, 64, G, a.dim), t(nb, 64, G, a.vdim)
        freq = torch.zeros(0, dtype=torch.float64, device="cuda")
        add("window_prep (value norm, cache)", "qk_norm_rope_cache", shape,
            lambda: K.C.window_prep(proj, meta.positions, meta.slot_mapping, freq, 1.0, None, None, 1e-6, kc, vc, q, asz, *MC._aside(None, T), True),
            2 * T * (al.rows + H * a.dim + G * (a.dim + a.vdim)))
        q2, k2, v2, qw = t(T, H, a.dim), t(T, G, a.dim), t(T, G, a.vdim), t(a.dim)
        add("qk_norm_rope_cache", "", shape, lambda: K.qk_norm_rope_cache(q2, k2, v2, qw, qw, meta.positions, 1e6, 1e-6, kc, vc, meta.slot_mapping),
            2 * (2 * q2.numel() + 5 * k2.numel()))
    w1 = torch.nn.Parameter(t(ds.beta_at + m.heads, D))
    for T in (1, 4):
        x, y, r2_ = t(T, D, dtype=torch.float32), t(T, D), t(T, D)
        for name, yn, n2 in (("factor, norm", None, nw), ("normed addend, norm", nw, nw), ("factor, no norm", None, None)):
            add(f"residual_linear ({name})", "add_rmsnorm_linear", f"{T} rows", lambda: MC.residual_linear(x, y, yn, 0.4, n2, 1e-6, w1), 2 * w1.numel())
        add("add_rmsnorm_linear", "", f"{T} rows", lambda: K.add_rmsnorm_linear(y, r2_, nw, 1e-6, w1), 2 * w1.numel())
    lg = t(64, cfg.vocab_size, dtype=torch.float32)
    add("softcap (64 rows of logits)", "swiglu", "64 rows", lambda: MC.softcap_(lg, 30.0, False), 8 * lg.numel())
    return out.rows


def main(a) -> int:
    from ..models.config import get_config
    from ..ops import build
    from ..ops import cuda as K

    torch.cuda.set_device(0)
    cfg = get_config(a.layered_model)
    moe = cfg.num_moe_layers > 0
    parts = build.serve_kind(cfg).split("_")
    base = get_config(a.layered_baseline or ("qwen3-30B-A3B" if moe else "nopelorn-4B-shape" if "delta" in parts else "qwen3-4B"))
    cfg = cfg.with_(num_layers=a.layers or (8 if moe else 12))
    base = base.with_(num_layers=len(cfg.runs()))      # (a layered baseline keeps its first layers)
    for c in (cfg, base):
        print(json.dumps(throughput(c)), flush=True)
        torch.cuda.empty_cache()
    kinds = {"delta": delta_kernels, "ssm": hybrid_kernels, "linear": latent_kernels, "attention": attention_kernels}
    for r in next(f for part, f in kinds.items() if part in parts)(cfg, base):
        print(json.dumps(r), flush=True)
    print(json.dumps({"kernel_error_flag": K.check_error_flag()}))
    return 0
