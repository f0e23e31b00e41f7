"""Checks shared by the CPU and the GPU tests of Nopelorn (device and dtype are arguments)."""
from __future__ import annotations

import torch

import layered_utils as U
import plain_nopelorn as plain

EPS = 1e-5


def config_a():
    """Every kind of layer; a layer on another's latents with its own window and head sizes; one layer without a feed-forward."""
    return plain.make_config([plain.lightning_spec(heads=2, dim=16, vdim=24), plain.latent_spec(window=19),
                              plain.latent_spec(heads=2, dim=16, vdim=16, window=37, kv_from=1, ff=56),
                              plain.lightning_spec(heads=3, dim=24, vdim=8, ff=None)])


def config_b():
    """Sizes that are no multiples of anything, single heads, a window of one token, no feed-forward anywhere but once."""
    return plain.make_config([plain.latent_spec(heads=1, dim=11, rot_dim=6, vdim=7, kv_rank=13, window=1, ff=None),
                              plain.lightning_spec(heads=1, dim=5, vdim=3, decay=[0.9], ff=19),
                              plain.latent_spec(heads=3, dim=10, rot_dim=2, vdim=9, kv_rank=21, window=23, ff=None)],
                             width=37, vocab=53, buckets=7, mul_prev=1, mul_cur=1)


def config_c():
    """Tensor-core sizes: two head groups, two column atoms, wide windows, 128-wide states."""
    return plain.make_config([plain.latent_spec(heads=20, dim=72, rot_dim=16, vdim=80, kv_rank=112, window=70, ff=256),
                              plain.lightning_spec(heads=2, dim=128, vdim=128, decay=[0.6, 0.999], ff=256),
                              plain.latent_spec(heads=5, dim=128, rot_dim=16, vdim=128, kv_rank=112, window=150, kv_from=0, ff=320),
                              plain.latent_spec(heads=17, dim=24, rot_dim=32, vdim=40, kv_rank=48, window=33, ff=None)],
                            width=256, vocab=300)


def sizes_for_all(engine_kw, cfg, T, patterns, tol, seed=0, gain=1.0):
    """One request in differently cut pieces against the plain model; every cut gives the same logits up to rounding."""
    W = plain.make_weights(cfg, seed, gain=gain)
    toks = U.tokens_for(cfg, T, seed)
    want = plain.run(cfg, W, toks)
    e = U.engine_for(cfg, W, **engine_kw)
    for p in patterns:
        got = U.feed_alone(e, toks, U.sizes_for(T, p))
        assert U.rel(got, want) < tol, (p, U.rel(got, want))
    return e


def mixed_batches(engine_kw, cfg, lengths, tol, seed=3):
    """Unequal requests together (pieces beside single tokens, some left out of steps), each against itself alone; pages and slots
    come from a pool that only fits by using them again."""
    W = plain.make_weights(cfg, seed)
    seqs = {f"r{i}": U.tokens_for(cfg, n, 10 + i) for i, n in enumerate(lengths)}
    e = U.engine_for(cfg, W, **engine_kw)
    schedule = U.random_schedule({n: len(s) for n, s in seqs.items()}, seed)
    out = U.feed_together(e, schedule, seqs)
    for n, s in seqs.items():
        want = plain.run(cfg, W, s)
        assert U.rel(out[n], want) < tol, (n, U.rel(out[n], want))
    assert e.allocator.num_free == engine_kw.get("blocks", 24) and e.states.num_free == engine_kw.get("slots", 4)


def window_edges(device, dtype, m, T, tol, portions, strength=16.0):
    """A query that points at one key: the oldest key of its window, the one just outside, one at a page border, the first token."""
    w, bs = m["mask"]["size"], 16
    for key, query in [(T - 1 - (w - 1), T - 1), (T - 1 - w, T - 1), (bs * 2 - 1, min(T - 1, bs * 2 + w // 2)), (bs * 2, bs * 2 + w - 1),
                       (0, w - 1), (0, w), (T - 1, T - 1)]:
        if not (0 <= key <= query < T):
            continue
        h, W = U.latent_case(m, T, seed=query)
        U.point_at(h, W, m, EPS, query, key, strength)
        want = plain.latent_attention(h, W, "x.", m, EPS, plain.latent_of(h, W, "x.", m, EPS))
        for sizes in portions:
            pages = U.Pages([T], bs, device)
            cache = U.latent_cache(m, pages, dtype)
            got = U.run_pieces(pages, [h], [[(0, n)] for n in U.sizes_for(T, sizes)], U.latent_fn(m, W, cache, dtype, device, EPS))[0]
            assert U.rel(got, want) < tol, (key, query, sizes, U.rel(got, want))
            assert U.rel(got[query:query + 1], want[query:query + 1]) < tol, (key, query, sizes)
        # the case tells the two sides of the edge apart: with a window one token wider or narrower the answer is another one
        if query - key in (w - 1, w):
            other = dict(m, mask={"size": w + 1 if query - key == w else w - 1})
            if other["mask"]["size"] > 0:
                off = plain.latent_attention(h, W, "x.", other, EPS, plain.latent_of(h, W, "x.", m, EPS))
                assert U.rel(off[query:query + 1], want[query:query + 1]) > 20 * tol


def sink_counts(device, dtype, m, T, tol):
    """A sink far above the scores drains the output, one far below changes nothing, and it counts once."""
    for value in (-30.0, 0.0, 6.0, 30.0):
        h, W = U.latent_case(m, T, seed=5)
        W["x.sink"] = torch.full_like(W["x.sink"], value)
        want = plain.latent_attention(h, W, "x.", m, EPS, plain.latent_of(h, W, "x.", m, EPS))
        for sizes in ([T], [1], [5, 23]):
            pages = U.Pages([T], 16, device)
            cache = U.latent_cache(m, pages, dtype)
            got = U.run_pieces(pages, [h], [[(0, n)] for n in U.sizes_for(T, sizes)], U.latent_fn(m, W, cache, dtype, device, EPS))[0]
            assert U.rel(got, want) < tol, (value, sizes, U.rel(got, want))


def linear_state(device, dtype, H, dk, dv, lengths, schedule, tol, decay=None, pull=None):
    """Linear attention over several sequences in pieces against one token after another.  `pull` = (write, read): the key and
    query of these two tokens of the first sequence are aligned and large, so that a state lost in between shows."""
    from miles_b200.ops import mixers as MX

    g = torch.Generator().manual_seed(1)
    decay = decay or [0.5 + 0.499 * (i + 1) / H for i in range(H)]
    C = H * (2 * dk + 2 * dv)
    xs = [torch.randn(n, C, generator=g).bfloat16().double() for n in lengths]
    if pull:
        a, b = pull
        row = 3 * torch.rand(H * dk, generator=g).double()
        xs[0][a, H * dk:2 * H * dk] = row.bfloat16().double()
        xs[0][b, : H * dk] = row.bfloat16().double()
    norm = (1 + 0.2 * torch.randn(H * dv, generator=g)).bfloat16().double()
    pages = U.Pages(lengths, 16, device)
    state = 100 * torch.randn(len(lengths), H, dk, dv, generator=g).to(device)      # slots that were used before
    dec = torch.tensor(decay, dtype=torch.float64).float().to(device)
    nw = norm.to(device=device, dtype=dtype)
    got = U.run_pieces(pages, xs, schedule, lambda x, m: MX.linear_state_attention(x.to(dtype), H, dk, dv, dec, state, m, nw, EPS))
    for x, y in zip(xs, got):
        q, k, v, gate = x.split([H * dk, H * dk, H * dv, H * dv], -1)
        o = plain.lightning_states(plain.silu(q).view(-1, H, dk), plain.silu(k).view(-1, H, dk), plain.silu(v).view(-1, H, dv),
                                   torch.tensor(decay, dtype=torch.float64)).reshape(len(x), H * dv)
        want = plain.rms(o, EPS) * norm / (1 + torch.exp(-gate))
        assert U.rel(y, want) < tol, U.rel(y, want)


def greedy(cfg, W, prompt, n):
    """Greedy continuation by the plain model and the margin of every choice."""
    toks, margins = list(prompt), []
    for _ in range(n):
        lg = plain.run(cfg, W, toks)[-1]
        top = lg.topk(2).values
        margins.append(float(top[0] - top[1]))
        toks.append(int(lg.argmax()))
    return toks[len(prompt):], margins
