"""Checks shared by the CPU and the GPU tests of Vozirax (device and dtype are arguments)."""
from __future__ import annotations

import math

import torch

import layered_utils as U
import plain_vozirax as plain
from plain_vozirax import attn, ff, layer, moe, ssm

EPS = 1e-5


def config_a():
    """Unlike layers of both kinds, every kind of feed-forward, a layer on another's keys and values with other constants of its own."""
    return plain.make_config([layer(ssm(), ff()), layer(attn(), moe()), layer(ssm(heads=4, vdim=12, state=20, groups=4, taps=2, norm_groups=1), None),
                              layer(attn(diff=0.6, coef=None, kv_from=1, scale=0.4), moe(experts=5, top=2, n=24, count=None)),
                              layer(ssm(heads=3, vdim=8, state=16, groups=1, taps=1, norm_groups=4), moe(count=8, keep=3, top=2))])


def config_b():
    """Sizes that are no multiples of anything, single heads, one expert, more taps; attention first."""
    return plain.make_config([layer(attn(heads=1, kv_heads=1, dim=7, vdim=5, diff=0.2, every=4), moe(experts=1, top=1, n=9, count=1, keep=1)),
                              layer(ssm(heads=1, vdim=9, state=5, groups=1, taps=6, norm_groups=1), ff(11)),
                              layer(ssm(heads=5, vdim=3, state=7, groups=5, taps=3, norm_groups=5), moe(experts=9, top=3, n=13, count=3, keep=2)),
                              layer(attn(heads=4, kv_heads=1, dim=10, vdim=11, diff=0.7), None)], width=37, vocab=53, logit_scale=2.5)


def config_c():
    """Tensor-core sizes: pairs of heads in a tile and single ones, group sizes of 2 to 24 query rows, one and two column atoms."""
    return plain.make_config([layer(ssm(heads=8, vdim=64, state=128, groups=2, taps=4, norm_groups=1), ff(96)),
                              layer(attn(heads=8, kv_heads=1, dim=64, vdim=128, every=30), moe(experts=16, top=4, n=64, count=4, keep=2)),
                              layer(ssm(heads=4, vdim=32, state=72, groups=1, taps=3, norm_groups=2), moe(experts=6, top=2, n=32, count=2, keep=1)),
                              layer(attn(heads=12, kv_heads=1, dim=32, vdim=64, diff=0.1, every=64), ff(160)),
                              layer(ssm(heads=3, vdim=104, state=40, groups=3, taps=4, norm_groups=3), None),
                              layer(attn(heads=8, kv_heads=1, dim=64, vdim=128, kv_from=1), moe(experts=12, top=1, n=96, count=3, keep=3))], width=256, vocab=300)


def close(got, want, tol, note=None):
    """Every row within `tol`.  In 16 bits the norms behind a difference or a gate can make much of little: where hardly anything is left
    to be normed, a row may be off by more.  (16-bit runs use weights without close calls between experts.)"""
    err = U.row_errors(got, want)
    few = max(1, int(0.02 * len(err))) if tol > 1e-3 and len(err) > 9 else 0
    assert float(err.sort().values[len(err) - 1 - few]) < tol and float(err.max()) < 4 * tol, (note, float(err.max()), tol)


def weights_for(engine_kw, cfg, seed):
    return plain.make_weights(cfg, seed, apart=engine_kw["dtype"] == torch.bfloat16)


def row_rel(got, want) -> float:
    """Largest error of a row relative to that row's or the rows' root mean square, whichever is larger."""
    got, want = got.double().cpu(), want.double().cpu()
    own = want.square().mean(-1).sqrt()
    return float(((got - want).square().mean(-1).sqrt() / torch.maximum(own, want.square().mean().sqrt())).max())


def sizes_for_all(engine_kw, cfg, T, patterns, tol, seed=0):
    """One request in differently cut pieces against the plain model."""
    W = weights_for(engine_kw, cfg, seed)
    toks = U.tokens_for(cfg, T, seed)
    want = plain.run(cfg, W, toks)
    e = U.engine_for(cfg, W, **engine_kw)
    for p in patterns:
        close(U.feed_alone(e, toks, U.sizes_for(T, p)), want, tol, p)
    return e


def mixed_batches(engine_kw, cfg, lengths, tol, seed=3):
    """Unequal requests together, each against itself alone; pages and slots only suffice by using them again."""
    W = weights_for(engine_kw, cfg, seed)
    seqs = {f"r{i}": U.tokens_for(cfg, n, 10 + i) for i, n in enumerate(lengths)}
    e = U.engine_for(cfg, W, prefix_cache=False, **engine_kw)
    out = U.feed_together(e, U.random_schedule({n: len(s) for n, s in seqs.items()}, seed), seqs)
    for n, s in seqs.items():
        close(out[n], plain.run(cfg, W, s), tol, n)
    assert e.allocator.num_free == engine_kw.get("blocks", 24) and (e.states is None or e.states.num_free == e.states.num_slots)


def exact(t):
    return t.bfloat16().double()


# ---- the state-space op ----------------------------------------------------------------------------------------------------------

def ssm_case(m, T, seed=0, keep=True):
    """(rows [z; x; B; C; dt] of a whole sequence, the mixer's vectors), bf16-exact.  `keep`: every second head hardly forgets."""
    g = torch.Generator().manual_seed(seed)
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    ch = H * V + 2 * G * N

    def rnd(*s, k=1.0, mean=0.0):
        return exact(mean + k * torch.randn(*s, generator=g))

    W = {"conv": rnd(ch, m["conv"], k=0.8), "conv.b": rnd(ch, k=0.2), "dt_bias": rnd(H, mean=-2.0, k=0.5), "A_log": rnd(H, mean=-1.0), "D": rnd(H)}
    if keep:
        W["A_log"][::2] = -9.0
    return rnd(T, H * V + ch + H), W


def ssm_parts(case, m):
    x, W = case
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    z, xbc, dt = x.split([H * V, H * V + 2 * G * N, H], -1)
    xs, B, C = plain.short_conv(xbc, W["conv"], W["conv.b"]).split([H * V, G * N, G * N], -1)
    return z, xs.unflatten(-1, (H, V)), B.unflatten(-1, (G, N)), C.unflatten(-1, (G, N)), plain.step_sizes(dt, W["dt_bias"])


def ssm_want(case, m):
    z, x, B, C, dt = ssm_parts(case, m)
    y = plain.recurrence(x, B, C, dt, case[1]["A_log"], case[1]["D"]).flatten(1)
    return y * z * torch.sigmoid(z)


def ssm_fn(m, case, pages, dtype, device, aside=None):
    """fn(rows, meta) → gated outputs through the package's op; states and rings were used before."""
    from miles_b200.ops import mixers as MX

    lay = MX.SsmLayout(m["heads"], m["vdim"], m["state"], m["groups"], m["conv"])
    g = torch.Generator().manual_seed(5)
    n = len(pages.slots)
    state = (50 * torch.randn(n, m["heads"], m["state"], m["vdim"], generator=g)).to(device)
    ring = (50 * torch.randn(n, m["conv"], lay.channels, generator=g)).to(device) if m["conv"] > 1 else None
    w = [case[1][k].to(device=device, dtype=dtype).contiguous() for k in ("conv", "conv.b", "dt_bias", "A_log", "D")]

    def fn(x, meta):
        wide = torch.full((len(x), -(-x.shape[1] // 8) * 8 + 8), 33.0, dtype=dtype, device=device)      # rows of a wider buffer
        wide[:, : x.shape[1]] = x.to(dtype)
        return MX.state_space(wide[:, : x.shape[1]], lay, *w, state, ring, meta, aside=aside)

    return fn


def run_ssm(cases, m, schedule, dtype, device, bs=16):
    pages = U.Pages([len(c[0]) for c in cases], bs, device)
    return U.run_pieces(pages, [c[0] for c in cases], schedule, ssm_fn(m, cases[0], pages, dtype, device))


def remembered(device, dtype, m, T, pairs, tol, portions):
    """One token's x stands out and a later token's C asks for its B: the state has to carry it there, over chunks, segments and pieces."""
    for key, query in pairs:
        case = ssm_case(m, T, seed=key)
        x, W = case
        H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
        W["conv"][H * V:, :-1] = 0                          # B and C of a token are its own
        W["conv"][H * V:, -1] = 1
        W["conv.b"][H * V:] = 0
        x[key, H * V: 2 * H * V] *= 40
        b0, c0 = 2 * H * V, 2 * H * V + G * N
        x[key, b0: c0] = exact(3 * x[key, b0: c0].sign())
        x[query, c0: c0 + G * N] = exact(2 * x[key, b0: c0])
        want = ssm_want(case, m)
        gone = x.clone()
        gone[key, H * V: 2 * H * V] = 0
        told = U.row_errors(ssm_want((gone, W), m)[query:query + 1], want[query:query + 1])
        assert query < key or float(told) > 6 * tol, (key, query, float(told))
        for sizes in portions:
            got = run_ssm([case], m, [[(0, n)] for n in U.sizes_for(T, sizes)], dtype, device)[0]
            assert row_rel(got, want) < tol, (key, query, sizes, row_rel(got, want))
            assert U.rel(got[query:query + 1], want[query:query + 1]) < tol, (key, query, sizes)


# ---- the attention op ----------------------------------------------------------------------------------------------------------

def attention_case(m, T, seed=0):
    """(rows [q; k; v; gate], the mixer's vectors), bf16-exact"""
    g = torch.Generator().manual_seed(seed)
    n = m["heads"] * 2 * m["dim"] + m["kv_heads"] * (2 * m["dim"] + m["vdim"]) + m["heads"]
    W = {k: exact(0.3 * torch.randn(m["dim"], generator=g)) for k in ("lq1", "lk1", "lq2", "lk2")}
    W.update({k: exact(1 + 0.2 * torch.randn(m["dim"], generator=g)) for k in ("q.norm", "k.norm")})
    return exact(torch.randn(T, n, generator=g)), W


def attention_split(x, m):
    return x.split([m["heads"] * 2 * m["dim"], m["kv_heads"] * 2 * m["dim"], m["kv_heads"] * m["vdim"], m["heads"]], -1)


def attention_want(case, m, sees_next=False):
    x, W = case
    q, k, v, gate = attention_split(x, m)
    k = plain.rms(k.unflatten(-1, (m["kv_heads"], 2, m["dim"])), EPS) * W["k.norm"]
    return plain.attend(plain.queries(q, W["q.norm"], m, EPS), k, v.unflatten(-1, (m["kv_heads"], m["vdim"])), gate,
                        plain.mix_weight(W, "", m["diff"]), m, EPS)


def point_at(case, m, query: int, key: int, key2: int):
    """The first map of every head of token `query` points at token `key`, the second at `key2`."""
    x, W = case
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    k = attention_split(x, m)[1].unflatten(-1, (G, 2, d))
    k = plain.rms(k, EPS) * W["k.norm"]
    q = torch.stack([k[key, :, 0], k[key2, :, 1]], 1).repeat_interleave(H // G, 0)      # [H, 2, d]
    x[query, : H * 2 * d] = exact((q / W["q.norm"]).flatten())


def attention_fn(m, case, caches, dtype, device, aside=None, writes=True):
    from miles_b200.ops import mixers as MX

    lay = MX.DifferentialLayout(m["heads"], m["kv_heads"], m["dim"], m["vdim"], writes)
    W = {k: t.to(device=device, dtype=dtype) for k, t in case[1].items()}
    lvec = torch.stack([W[k] for k in ("lq1", "lk1", "lq2", "lk2")])
    t = m.get("q_temp")
    return lambda x, meta: MX.differential_attention(x.to(dtype), lay, *caches, meta, scale=m["scale"], diff=m["diff"],
                                                     temperature=(t["coef"], t["every"]) if t else None, lvec=lvec, q_norm=W["q.norm"],
                                                     k_norm=W["k.norm"] if writes else None, eps=EPS, aside=aside)


def attention_caches(m, pages, dtype):
    """Pages that were used before: what lies outside a sequence's own positions must not matter."""
    g = torch.Generator().manual_seed(9)
    return tuple((50 * torch.randn(pages.num_blocks, pages.bs, m["kv_heads"], n, generator=g)).to(dtype).to(pages.device) for n in (2 * m["dim"], m["vdim"]))


def run_attention(cases, m, schedule, dtype, device, bs=16):
    pages = U.Pages([len(c[0]) for c in cases], bs, device)
    return U.run_pieces(pages, [c[0] for c in cases], schedule, attention_fn(m, cases[0], attention_caches(m, pages, dtype), dtype, device))


def sharp(**kw):
    """A mixer whose queries, pointed at a key, see little else."""
    m = attn(**kw)
    m["scale"] = 10.0 / m["dim"]
    return m


def pointed(device, dtype, m, T, pairs, tol, portions, bs=16):
    """Maps that point at single keys: far ones, the first, page borders, itself, and one token too far (which must stay unseen)."""
    for query, key, key2 in pairs:
        case = attention_case(m, T, seed=query + key)
        point_at(case, m, query, key, key2)
        want = attention_want(case, m)
        if key <= query:                                    # the row tells the two maps and its key apart
            other = attention_case(m, T, seed=query + key)
            point_at(other, m, query, (key + 1) % (query + 1), key2)
            assert query == 0 or U.rel(attention_want(other, m)[query:query + 1], want[query:query + 1]) > 3 * tol
        for sizes in portions:
            got = run_attention([case], m, [[(0, n)] for n in U.sizes_for(T, sizes)], dtype, device, bs)[0]
            close(got, want, tol, (query, key, sizes))
            assert U.rel(got[query:query + 1], want[query:query + 1]) < tol, (query, key, sizes)


# ---- choice of experts, experts, sums -----------------------------------------------------------------------------------------------

CHOICES = [(1, 1, 1, 1, 1), (5, 12, 2, 3, 2), (70, 128, 8, 8, 4), (9, 300, 6, 30, 7), (3, 33, 4, 11, 3), (4, 6, 2, 6, 3), (6, 512, 8, 256, 20), (7, 40, 5, 1, 1),
           (8, 64, 3, 2, 1)]


def choice(device, dtype, T, E, k, count, keep, run):
    """`run(aside)` chooses on the way; against the plain statement.  Corrections push many choice scores below zero."""
    from miles_b200.ops import mixers as MX

    g = torch.Generator().manual_seed(E + T)
    z = 1.5 * torch.randn(T, E, generator=g)
    corr = exact(-0.6 + 0.4 * torch.randn(E, generator=g))
    a = MX.Aside(logits=z.to(device), top=k, routing=MX.Routing(count, keep, 1.7), correction=corr.to(device=device, dtype=dtype))
    run(a)
    idx, w = plain.choose(z.double(), corr, {"top": k, "scale": 1.7, "groups": {"count": count, "keep": keep}})
    assert torch.equal(a.index.cpu().long(), idx) and torch.allclose(a.weights.cpu().double(), w, atol=2e-6 if dtype == torch.float32 else 2e-5)
    # equal scores everywhere: the lowest groups and experts
    a = MX.Aside(logits=torch.zeros(T, E, device=device), top=k, routing=MX.Routing(count, keep, 2.0))
    run(a)
    if device != "cpu":
        assert torch.equal(a.index.cpu(), torch.arange(k).expand(T, k).int())
    assert torch.allclose(a.weights.cpu(), torch.full((T, k), 2.0 / k))


def experts(device, dtype, T, E, k, D, F, tol, skew=False):
    """Ungated experts on given choices, added with a scale per channel, against the plain statement."""
    from miles_b200.ops import mixers as MX

    g = torch.Generator().manual_seed(T + E)
    h, w1, w2, s = (exact(c * torch.randn(*sh, generator=g)) for c, sh in ((1, (T, D)), (1.5 / D ** 0.5, (E, F, D)), (1 / F ** 0.5, (E, D, F)), (1, (D,))))
    idx = torch.rand(T, E, generator=g).topk(k, -1).indices
    if skew:
        idx[:, 0] = E - 1
        idx[:, 1:] = torch.rand(T, E - 1, generator=g).topk(k - 1, -1).indices
    w = torch.rand(T, k, generator=g).double()
    W = {f"e{e}.{n}": t for e in range(E) for n, t in (("up", w1[e]), ("down", w2[e]))}
    want = s * torch.stack([sum(w[t, j] * plain.expert(h[t], W, f"e{int(e)}") for j, e in enumerate(idx[t])) for t in range(T)])

    def put(t, dt=dtype):
        return t.to(device=device, dtype=dt).contiguous()

    with torch.no_grad():
        a = MX.routed_experts(put(h), put(w1), put(w2), put(w, torch.float32), put(idx, torch.int32), ungated=True)
        a.scale = put(s)
        x = torch.zeros(T, D, dtype=torch.float32, device=device)
        to = torch.empty_like(x)
        assert MX.sum_norm(x, to, [a], None, None, 1e-6) is None
    assert U.rel(to, want) < tol, U.rel(to, want)


def sums(device, dtype, T, D, tol):
    """Scaled addends, two norms with weights around zero, a gain."""
    from miles_b200.ops import mixers as MX

    g = torch.Generator().manual_seed(T + D)

    def rnd(*s, dt=dtype, k=1.0):
        return (k * torch.randn(*s, generator=g)).to(dt).to(device)

    x, a, b, rows = rnd(T, D, dt=torch.float32), rnd(T, D), rnd(T, D), rnd(3 * T, D)
    s1, s2, n1, n2 = rnd(D), rnd(D), rnd(D, k=0.2), rnd(D, k=0.2)
    adds = [([], x.double()), ([MX.Addend(a, scale=s1)], x.double() + a.double() * s1.double()),
            ([MX.Addend(a, scale=s1), MX.Addend(b, scale=s2)], x.double() + a.double() * s1.double() + b.double() * s2.double())]
    if device != "cpu":
        w, dst = torch.rand(T, 3, generator=g).to(device), torch.randperm(3 * T, generator=g).int().to(device)
        dst[0] = -1
        gathered = (w.double()[..., None] * torch.where(dst[:, None] >= 0, rows.double()[dst.long()], 0.0).view(T, 3, D)).sum(1)
        adds.append(([MX.Addend(a, scale=s1), MX.Addend(rows, w, dst, s2)], x.double() + a.double() * s1.double() + gathered * s2.double()))
    for add, want in adds:
        to = torch.empty_like(x)
        h, h2 = MX.sum_norm(x, to, add, None, n1, 1e-5, shift=1.0, gain=0.4, nw2=n2, two=True)
        assert U.rel(to, want) < 1e-6
        n = plain.rms(want, 1e-5)
        assert U.rel(h, n * (1 + n1.double()) * 0.4) < tol and U.rel(h2, n * (1 + n2.double()) * 0.4) < tol


def embedding(device, dtype, width, tol):
    from miles_b200.ops import mixers as MX

    pos = torch.tensor([0, 1, 2, 77, 4095, 30000, 1000003])
    embed = torch.zeros(5, width, dtype=dtype, device=device)
    freq = torch.tensor([10000.0 ** (-2 * i / width) for i in range((width + 1) // 2)], dtype=torch.float64, device=device)
    x, _ = MX.bigram_embedding(torch.zeros(7, dtype=torch.int32, device=device), torch.full((7,), -1, dtype=torch.int32, device=device), embed,
                               positions=pos.int().to(device), freq=freq)
    want = torch.stack([plain.place_vectors(1, width)[0] * 0 + torch.tensor(
        [math.cos(p * 10000.0 ** (-(c - 1) / width)) if c % 2 else math.sin(p * 10000.0 ** (-c / width)) for c in range(width)]) for p in pos.tolist()])
    assert x.dtype == torch.float32 and float((x.cpu().double() - want).abs().max()) < tol


def greedy(cfg, W, prompt, n):
    """Greedy continuation by the plain model."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(plain.run(cfg, W, toks)[-1].argmax()))
    return toks[len(prompt):]
