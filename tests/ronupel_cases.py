"""Checks shared by the CPU and the GPU tests of Ronupel (device and dtype are arguments)."""
from __future__ import annotations

import torch

import layered_utils as U
import plain_ronupel as plain

EPS = 1e-5


def config_a():
    """Unlike layers: windows, kept tokens, head counts and value sizes of their own, one layer without a feed-forward, one without a
    shared expert, three passes over the middle."""
    return plain.make_config([plain.layer_spec(),
                              plain.layer_spec(heads=4, kv_heads=4, dim=16, vdim=16, window=37, keep=0, experts=3, top=3, ff=24, shared=0, factor=1.0),
                              plain.layer_spec(heads=3, kv_heads=1, dim=32, vdim=24, rot=32, window=11, keep=20, experts=0),
                              plain.layer_spec(window=30, keep=2, experts=7, top=1, ff=40, shared=16)], loop=(1, 3, 3))


def config_b():
    """Sizes that are no multiples of anything, single heads, a window of one token, one expert, the loop at the start."""
    return plain.make_config([plain.layer_spec(heads=1, kv_heads=1, dim=7, vdim=5, rot=2, window=1, keep=3, experts=1, top=1, ff=9, shared=3),
                              plain.layer_spec(heads=5, kv_heads=1, dim=10, vdim=9, rot=6, window=23, keep=1, experts=3, top=2, ff=11, shared=13)],
                             width=37, vocab=53, loop=(0, 1, 2))


def config_c():
    """Tensor-core sizes: groups of 1, 3, 5 and 16 heads, one and two column atoms, windows and kept tokens beyond a tile, no loop; a layer
    that sees everything."""
    return plain.make_config([plain.layer_spec(heads=5, kv_heads=5, dim=72, vdim=80, rot=40, window=70, keep=66, experts=6, ff=64, shared=128),
                              plain.layer_spec(heads=15, kv_heads=3, dim=128, vdim=64, rot=128, window=150, keep=10, experts=9, top=4, ff=32, shared=0),
                              plain.layer_spec(heads=16, kv_heads=1, dim=40, vdim=128, rot=24, window=0, experts=8, top=2, ff=96, shared=96),
                              plain.layer_spec(heads=6, kv_heads=2, dim=16, vdim=24, rot=16, window=33, keep=130, experts=0)],
                             width=256, vocab=300)


def close(got, want, tol, note=None):
    """Every row within `tol`; with routed experts in 16 bits a token now and then chooses another expert where two are equally good, so a
    few rows may be off by more."""
    err = U.row_errors(got, want)
    few = max(2, int(0.03 * len(err))) if tol > 1e-3 else 0
    assert float(err.sort().values[len(err) - 1 - few if len(err) > few else 0]) < tol and float(err.max()) < 12 * tol, (note, float(err.max()), tol)


def sizes_for_all(engine_kw, cfg, T, patterns, tol, seed=0):
    """One request in differently cut pieces against the plain model."""
    W = plain.make_weights(cfg, seed)
    toks = U.tokens_for(cfg, T, seed)
    want = plain.run(cfg, W, toks)
    e = U.engine_for(cfg, W, **engine_kw)
    for p in patterns:
        close(U.feed_alone(e, toks, U.sizes_for(T, p)), want, tol, p)
    return e


def mixed_batches(engine_kw, cfg, lengths, tol, seed=3):
    """Unequal requests together, each against itself alone; pages come from a pool that only fits by using them again."""
    W = plain.make_weights(cfg, seed)
    seqs = {f"r{i}": U.tokens_for(cfg, n, 10 + i) for i, n in enumerate(lengths)}
    e = U.engine_for(cfg, W, prefix_cache=False, **engine_kw)
    out = U.feed_together(e, U.random_schedule({n: len(s) for n, s in seqs.items()}, seed), seqs)
    for n, s in seqs.items():
        close(out[n], plain.run(cfg, W, s), tol, n)
    assert e.allocator.num_free == engine_kw.get("blocks", 24)


# ---- the attention op ----------------------------------------------------------------------------------------------------------

def attention_case(m, T, seed=0):
    """(rows [q; k; v] of a whole sequence, bf16-exact; query norm, key norm, sink)"""
    g = torch.Generator().manual_seed(seed)
    nq, nk, nv = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]

    def exact(t):
        return t.bfloat16().double()

    return (exact(torch.randn(T, nq + nk + nv, generator=g)), exact(1 + 0.2 * torch.randn(nq, generator=g)),
            exact(1 + 0.2 * torch.randn(nk, generator=g)), exact(torch.randn(m["heads"], generator=g)))


def point_at(case, m, query: int, key: int):
    """Make every head's query of token `query` parallel, after norm and rotation, to its key of token `key`."""
    x, qn, kn, _ = case
    nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
    k = plain.prepared(x[key:key + 1, nq:nq + nk], kn, m["kv_heads"], torch.tensor([key]), m, EPS)
    q = plain.rotate(k.repeat_interleave(m["heads"] // m["kv_heads"], 1), torch.tensor([query]), m.get("rot"), back=True)
    x[query, :nq] = (q.flatten() / qn).bfloat16().double()


def attention_want(case, m):
    x, qn, kn, sink = case
    nq, nk = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
    pos = torch.arange(len(x))
    return plain.attend(plain.prepared(x[:, :nq], qn, m["heads"], pos, m, EPS), plain.prepared(x[:, nq:nq + nk], kn, m["kv_heads"], pos, m, EPS),
                        x[:, nq + nk:].unflatten(-1, (m["kv_heads"], m["vdim"])), sink, m)


def attention_fn(m, case, caches, dtype, device):
    """fn(rows, meta) → attention output through the package's op, into rows of a wider buffer."""
    from miles_b200.models.ronupel import _mixer
    from miles_b200.ops import mixers as MX

    s = _mixer("attention", m)
    freq, mag = s.rotary.table() if s.rotary else ([], 1.0)
    lay = MX.AttentionLayout(s.heads, s.kv_heads, s.dim, s.vdim, 2 * len(freq), s.window, s.keep_first)
    qn, kn, sink = (t.to(device=device, dtype=dtype) for t in case[1:])
    freq = torch.tensor(freq, dtype=torch.float64, device=device)

    def fn(x, meta):
        out = torch.full((len(x), s.heads * s.vdim + 8), 77.0, dtype=dtype, device=device)
        MX.windowed_attention(x.to(dtype), lay, *caches, meta, out[:, :-8], freq=freq, magnitude=mag, scale=s.scale, sink=sink, q_norm=qn, k_norm=kn,
                              eps=EPS)
        assert bool((out[:, -8:] == 77).all())
        return out[:, :-8]

    return fn


def attention_caches(m, pages, dtype):
    """Pages that were used before: what lies outside a sequence's own positions must not matter."""
    g = torch.Generator().manual_seed(9)
    return tuple((50 * torch.randn(pages.num_blocks, pages.bs, m["kv_heads"], n, generator=g)).to(dtype).to(pages.device) for n in (m["dim"], m["vdim"]))


def run_attention(cases, m, schedule, dtype, device, bs=16):
    pages = U.Pages([len(c[0]) for c in cases], bs, device)
    return U.run_pieces(pages, [c[0] for c in cases], schedule, attention_fn(m, cases[0], attention_caches(m, pages, dtype), dtype, device))


def edges(device, dtype, m, T, tol, portions, bs=16):
    """A query that points at one key, on either side of every edge: the oldest key of its window and the one before, the last kept
    token and the next, the first token, a page border, itself."""
    w, k = m["mask"]["size"], m["mask"]["keep_first"]
    far = T - 1
    wanted = {(far - w + 1, far), (far - w, far), (k - 1, far), (k, far), (0, far), (k - 1, k + w - 1), (k, k + w - 1), (k, k + w), (bs - 1, bs + 3),
              (2 * bs, 2 * bs + w - 1), (0, w - 1), (0, w), (far, far), (0, 0)}
    told = 0
    for key, query in sorted(wanted):
        if not 0 <= key <= query < T:
            continue
        case = attention_case(m, T, seed=query)
        point_at(case, m, query, key)
        want = attention_want(case, m)
        for sizes in portions:
            got = run_attention([case], m, [[(0, n)] for n in U.sizes_for(T, sizes)], dtype, device, bs)[0]
            assert U.rel(got, want) < tol, (key, query, sizes, U.rel(got, want))
            assert U.rel(got[query:query + 1], want[query:query + 1]) < tol, (key, query, sizes)
        # the case tells both sides of its edge apart: with that edge one token over, the answer is another one
        for other in ({"size": w + 1, "keep_first": k}, {"size": w - 1, "keep_first": k}, {"size": w, "keep_first": k + 1}, {"size": w, "keep_first": k - 1}):
            if other["size"] > 0 and other["keep_first"] >= 0 and plain.visible(query, key, other) != plain.visible(query, key, m["mask"]):
                off = attention_want(case, dict(m, mask=other))
                assert U.rel(off[query:query + 1], want[query:query + 1]) > 10 * tol
                told += 1
    assert told >= 3


def sinks(device, dtype, m, T, tol):
    """A sink far above the scores drains the output, one far below changes nothing, and it counts once."""
    for value in (-30.0, 0.0, 6.0, 30.0):
        case = attention_case(m, T, 5)
        case[3].fill_(value)
        want = attention_want(case, m)
        for sizes in ([T], [1], [5, 23]):
            got = run_attention([case], m, [[(0, n)] for n in U.sizes_for(T, sizes)], dtype, device)[0]
            assert U.rel(got, want) < tol, (value, sizes, U.rel(got, want))


# ---- experts ---------------------------------------------------------------------------------------------------------------------

def experts(device, dtype, T, E, k, D, F, tol, skew=False):
    """Routed experts on given choices, and the choice itself, against the plain statements."""
    from miles_b200.ops import mixers as MX

    g = torch.Generator().manual_seed(T + E)

    def exact(*s, k=1.0):
        return (k * torch.randn(*s, generator=g)).bfloat16().double()

    h, w13, w2 = exact(T, D), exact(E, 2 * F, D, k=1.5 / D ** 0.5), exact(E, D, F, k=1 / F ** 0.5)
    z = exact(T, E, k=2.0)
    if skew:                                       # everybody's first choice is the last expert
        z[:, E - 1] += 30
    idx, w = plain.choose(z, k)
    W = {f"e{e}.{n}": t for e in range(E) for n, t in (("gate", w13[e, :F]), ("up", w13[e, F:]), ("down", w2[e]))}
    want = torch.stack([sum(w[t, j] * plain.expert(h[t], W, f"e{int(e)}", 1.2) for j, e in enumerate(idx[t])) for t in range(T)])

    def put(t, dt=dtype):
        return t.to(device=device, dtype=dt).contiguous()

    with torch.no_grad():
        a = MX.routed_experts(put(h), put(w13), put(w2), put(w, torch.float32), put(idx, torch.int32), 1.2, 1.702)
        x = torch.zeros(T, D, dtype=torch.float32, device=device)
        to = torch.empty_like(x)
        assert MX.sum_norm(x, to, [a], None, None, 1e-6) is None
    assert U.rel(to, want) < tol, U.rel(to, want)


def greedy(cfg, W, prompt, n):
    """Greedy continuation by the plain model."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(plain.run(cfg, W, toks)[-1].argmax()))
    return toks[len(prompt):]
