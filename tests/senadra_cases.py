"""Checks shared by the CPU and the GPU tests of Senadra (device and dtype are arguments)."""
from __future__ import annotations

import torch

import layered_utils as U
import plain_senadra as plain
from plain_senadra import attn, delta, latent, layer

EPS = 1e-5


def config_a():
    """All three mixers, a layer without feed-forward, one on another's keys and values with chunks of its own, one tap."""
    return plain.make_config([layer(delta()), layer(attn()), layer(latent(), None), layer(attn(heads=4, size=13, scale=0.4, kv_from=1), 40),
                              layer(delta(heads=3, kv_heads=1, dim=8, vdim=12, conv=1, decay_rank=5, gate_rank=9))])


def config_b():
    """Sizes that are no multiples of anything, single heads, more taps; attention first."""
    return plain.make_config([layer(attn(heads=1, kv_heads=1, dim=7, vdim=5, size=9), 11), layer(latent(2, 5, 6, 3, 13, 11), 9),
                              layer(delta(1, 1, 9, 5, 6, 3, 4), None), layer(delta(4, 4, 6, 7, 2, 1, 1), 13),
                              layer(attn(heads=3, kv_heads=1, dim=7, vdim=5, size=31, kv_from=None), None)], width=37, vocab=53, mult=1.0, side=5, softcap=30.0)


def config_c():
    """Tensor-core sizes: whole and partial tiles, groups of 1 to 12 query heads, chunks shorter and longer than a tile of keys."""
    return plain.make_config([layer(delta(4, 2, 128, 128, 4, 32, 64), 96), layer(attn(8, 2, 64, 128, size=70), 160), layer(latent(4, 128, 64, 128, 256, 96), 96),
                              layer(delta(2, 2, 72, 104, 3, 16, 16), None), layer(attn(24, 2, 64, 128, size=150, kv_from=1), 64),
                              layer(attn(2, 2, 104, 40, size=33), 96)], width=256, vocab=300, side=40)


def close(got, want, tol, note=None):
    """Every row within `tol`.  In 16 bits the gated norm of a state's outputs can make much of little: a few rows may be off by more."""
    err = U.row_errors(got, want)
    few = max(1, int(0.02 * len(err))) if tol > 1e-3 and len(err) > 9 else 0
    assert float(err.sort().values[len(err) - 1 - few]) < tol and float(err.max()) < 4 * tol, (note, float(err.max()), tol)


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
    """Unequal requests together, each against itself alone; pages and slots only suffice by using them again."""
    W = plain.make_weights(cfg, seed)
    seqs = {f"r{i}": U.tokens_for(cfg, n, 10 + i) for i, n in enumerate(lengths)}
    e = U.engine_for(cfg, W, prefix_cache=False, **engine_kw)
    out = U.feed_together(e, U.random_schedule({n: len(s) for n, s in seqs.items()}, seed), seqs)
    for n, s in seqs.items():
        close(out[n], plain.run(cfg, W, s), tol, n)
    assert e.allocator.num_free == engine_kw.get("blocks", 24) and e.states.num_free == e.states.num_slots


def exact(t):
    return t.bfloat16().double()


def row_rel(got, want) -> float:
    """Largest error of a row relative to that row's or the rows' root mean square, whichever is larger."""
    got, want = got.double().cpu(), want.double().cpu()
    own = want.square().mean(-1).sqrt()
    return float(((got - want).square().mean(-1).sqrt() / torch.maximum(own, want.square().mean().sqrt())).max())


def whole(x, dtype, device):
    """Rows as part of a wider buffer."""
    wide = torch.full((len(x), -(-x.shape[1] // 8) * 8 + 8), 33.0, dtype=dtype, device=device)
    wide[:, : x.shape[1]] = x.to(dtype)
    return wide[:, : x.shape[1]]


# ---- the delta rule -----------------------------------------------------------------------------------------------------------------

def delta_case(m, T, seed=0, forget=False):
    """(rows [q; k; v; decay latent; gate latent; β] of a sequence, the mixer's vectors), bf16-exact.  `forget`: channels that lose far more than
    32-bit exponents hold within a few tokens, beside others that lose nothing."""
    g = torch.Generator().manual_seed(seed)
    H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def rnd(*s, k=1.0, mean=0.0):
        return exact(mean + k * torch.randn(*s, generator=g))

    W = {f"{n}.conv": rnd(rows, m["conv"], k=0.8) for n, rows in (("q", G * K), ("k", G * K), ("v", H * V))}
    W.update({"a2": rnd(H * K, m["decay_rank"], k=m["decay_rank"] ** -0.5), "g2": rnd(H * V, m["gate_rank"], k=m["gate_rank"] ** -0.5),
              "A_log": rnd(H, mean=-2.0), "dt_bias": rnd(H * K, mean=-2.0), "norm": rnd(V, mean=1.0, k=0.2)})
    W["A_log"][::2] = -6.0
    if forget:
        W["A_log"][:] = 3.0
        W["dt_bias"] = exact(torch.where(torch.rand(H * K, generator=g) < 0.3, 3.0, -9.0).double())
        W["a2"] *= 0.25
    return rnd(T, 2 * G * K + H * V + m["decay_rank"] + m["gate_rank"] + H), W


def delta_split(x, m):
    G, K, HV = m["kv_heads"], m["dim"], m["heads"] * m["vdim"]
    return x.split([G * K, G * K, HV, m["decay_rank"], m["gate_rank"], m["heads"]], -1)


def delta_want(case, m):
    x, W = case
    H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v, a, gate, b = delta_split(x, m)
    q, k, v = (plain.short_conv(t, W[n + ".conv"]) for n, t in (("q", q), ("k", k), ("v", v)))
    q, k = plain.unit(q.unflatten(-1, (G, K))) / K ** 0.5, plain.unit(k.unflatten(-1, (G, K)))
    o = plain.delta_rule(q, k, v.unflatten(-1, (H, V)), plain.log_decays(a @ W["a2"].T, W["A_log"], W["dt_bias"]), plain.sigmoid(b))
    return (plain.rms(o, EPS) * W["norm"]).flatten(1) * plain.sigmoid(gate @ W["g2"].T)


def delta_fn(m, case, pages, dtype, device):
    """fn(rows, meta) → outputs through the package's op; states and rings were used before."""
    from miles_b200.ops import mixers as MX

    lay = MX.DeltaLayout(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], m["decay_rank"], m["gate_rank"])
    g = torch.Generator().manual_seed(5)
    n = len(pages.slots)
    state = (50 * torch.randn(n, m["heads"], m["dim"], m["vdim"], generator=g)).to(device)
    ring = (50 * torch.randn(n, m["conv"], lay.channels, generator=g)).to(device) if m["conv"] > 1 else None
    W = {k: t.to(device=device, dtype=dtype).contiguous() for k, t in case[1].items()}
    conv = torch.cat([W["q.conv"], W["k.conv"], W["v.conv"]])

    def fn(x, meta):
        with torch.no_grad():
            return MX.delta_rule(whole(x, dtype, device), lay, conv, W["a2"], W["g2"], W["A_log"], W["dt_bias"], W["norm"], state, ring, meta, EPS)

    return fn


def run_delta(cases, m, schedule, dtype, device, bs=16):
    pages = U.Pages([len(c[0]) for c in cases], bs, device)
    return U.run_pieces(pages, [c[0] for c in cases], schedule, delta_fn(m, cases[0], pages, dtype, device))


def remembered(device, dtype, m, T, pairs, tol, portions):
    """One token's value stands out and a later token's query asks for its key; the tokens between hardly write.  The state has to carry
    it there, over chunks, pieces and decode steps."""
    for key, query in pairs:
        case = delta_case(m, T, seed=key)
        x, W = case
        G, K, HV = m["kv_heads"], m["dim"], m["heads"] * m["vdim"]
        for n in ("q.conv", "k.conv"):
            W[n][:, :-1] = 0                                # queries and keys are their token's own
            W[n][:, -1] = 1
        W["A_log"][:] = -8.0
        x[key, 2 * G * K: 2 * G * K + HV] *= 20
        x[:, -m["heads"]:] = -7.0
        x[key, -m["heads"]:] = 4.0
        x[key, G * K: 2 * G * K] = exact(3 * torch.rand(G * K, generator=torch.Generator().manual_seed(query)))      # past the silu
        x[query, : G * K] = x[key, G * K: 2 * G * K]
        want = delta_want(case, m)
        gone = x.clone()
        gone[key, 2 * G * K: 2 * G * K + HV] *= -1
        told = U.row_errors(delta_want((gone, W), m)[query:query + 1], want[query:query + 1])
        assert float(told) > 6 * tol, (key, query, float(told))
        for sizes in portions:
            got = run_delta([case], m, [[(0, n)] for n in U.sizes_for(T, sizes)], dtype, device)[0]
            assert U.rel(got[query:query + 1], want[query:query + 1]) < tol, (key, query, sizes, U.rel(got[query:query + 1], want[query:query + 1]))


# ---- chunked attention ----------------------------------------------------------------------------------------------------------------

def attention_case(m, T, seed=0):
    """(rows [q; k; v; gate], {r1, r2}), bf16-exact"""
    g = torch.Generator().manual_seed(seed)
    n = m["heads"] * m["dim"] + m["kv_heads"] * (m["dim"] + m["vdim"]) + m["heads"] * m["vdim"]
    return exact(torch.randn(T, n, generator=g)), {k: exact(torch.rand(m["heads"], generator=g)) for k in ("r1", "r2")}


def attention_split(x, m):
    return x.split([m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]], -1)


def attention_want(case, m, off=0):
    x, W = case
    q, k, v, gate = attention_split(x, m)
    v = plain.rms(v.unflatten(-1, (m["kv_heads"], m["vdim"])), EPS)
    o = plain.attend(q.unflatten(-1, (m["heads"], m["dim"])), k.unflatten(-1, (m["kv_heads"], m["dim"])), v, W["r1"], W["r2"], m, off)
    return o * plain.sigmoid(gate)


def attention_caches(m, pages, dtype):
    """Pages that were used before: what lies outside a sequence's own positions must not matter."""
    g = torch.Generator().manual_seed(9)
    return tuple((50 * torch.randn(pages.num_blocks, pages.bs, m["kv_heads"], n, generator=g)).to(dtype).to(pages.device) for n in (m["dim"], m["vdim"]))


def attention_fn(m, case, caches, dtype, device, writes=True):
    from miles_b200.ops import mixers as MX

    lay = MX.AttentionLayout(m["heads"], m["kv_heads"], m["dim"], m["vdim"], 0, 0, 0, m["mask"]["size"], writes, True)
    r = [case[1][k].to(device=device, dtype=dtype) for k in ("r1", "r2")]
    freq = torch.zeros(0, dtype=torch.float64, device=device)
    HV = m["heads"] * m["vdim"]

    def fn(x, meta):
        x = whole(x, dtype, device)
        out = torch.empty(len(x), HV, dtype=dtype, device=device)
        MX.windowed_attention(x, lay, *caches, meta, out, freq=freq, magnitude=1.0, scale=m["scale"], sink=None, q_norm=None, k_norm=None, eps=EPS,
                              bias=r, gate=x[:, lay.rows: lay.rows + HV])
        return out

    return fn


def run_attention(cases, m, schedule, dtype, device, bs=16):
    pages = U.Pages([len(c[0]) for c in cases], bs, device)
    return U.run_pieces(pages, [c[0] for c in cases], schedule, attention_fn(m, cases[0], attention_caches(m, pages, dtype), dtype, device))


def point_at(x, m, query: int, key: int):
    """Every head of token `query` points at token `key`: that score stands out by far."""
    k = attention_split(x, m)[1][key].unflatten(0, (m["kv_heads"], m["dim"])).repeat_interleave(m["heads"] // m["kv_heads"], 0)
    x[query, : m["heads"] * m["dim"]] = exact((12.0 / m["scale"] * k / k.square().sum(-1, keepdim=True)).flatten())


def pointed(device, dtype, m, T, pairs, tol, portions, bs=16):
    """Queries that point at single keys: the first and the last of a chunk, the last one of the chunk before (which must stay unseen), page
    borders, themselves."""
    size = m["mask"]["size"]
    for query, key in pairs:
        case = attention_case(m, T, seed=query + key)
        point_at(case[0], m, query, key)
        want = attention_want(case, m)
        start = query // size * size
        if size > 1 and key in (start, start - 1) and key < query:      # a chunk that starts one token off would show in the row
            moved = attention_want(case, m, off=-1 if key == start else 1)
            assert U.rel(moved[query:query + 1], want[query:query + 1]) > 3 * tol, (query, key)
        for sizes in portions:
            got = run_attention([case], m, [[(0, n)] for n in U.sizes_for(T, sizes)], dtype, device, bs)[0]
            assert U.rel(got, want) < tol, (query, key, sizes, U.rel(got, want))
            assert U.rel(got[query:query + 1], want[query:query + 1]) < tol, (query, key, sizes)


def edge_pairs(size, T):
    """(query, key) at a chunk's first and last token and around both, and far apart."""
    out = [(0, 0), (T - 1, T - 1)]
    for c in range(size, T, size):
        out += [(c, c - 1), (c, c), (min(c + size, T) - 1, c), (min(c + size, T) - 1, c - 1), (c - 1, c - size)]
    return [p for p in out if p[1] >= 0]


# ---- latent attention -------------------------------------------------------------------------------------------------------------------

def latent_case(m, T, seed=0):
    """(rows [latent; rotated key part], queries, gate, the mixer's weights), bf16-exact"""
    g = torch.Generator().manual_seed(seed)
    H, r = m["heads"], m["kv_rank"]

    def rnd(*s, k=1.0, mean=0.0):
        return exact(mean + k * torch.randn(*s, generator=g))

    W = {"dkv.norm": rnd(r, mean=1.0, k=0.2), "uk": rnd(H * m["dim"], r, k=r ** -0.5), "uv": rnd(H * m["vdim"], r, k=r ** -0.5)}
    return torch.cat([rnd(T, r + m["rot_dim"]), rnd(T, H * (m["dim"] + m["rot_dim"])), rnd(T, H * m["vdim"])], -1), W


def latent_want(case, m):
    x, W = case
    c, kr, q, gate = x.split([m["kv_rank"], m["rot_dim"], m["heads"] * (m["dim"] + m["rot_dim"]), m["heads"] * m["vdim"]], -1)
    c = plain.rms(c, EPS) * W["dkv.norm"]
    return plain.latent_heads(q.unflatten(-1, (m["heads"], -1)), c, kr, W, "", m) * plain.sigmoid(gate)


def point_latent(case, m, query: int, key: int):
    """The unrotated query of token `query` is parallel to the unrotated key of token `key` in every head."""
    x, W = case
    H, d = m["heads"], m["dim"]
    k = ((plain.rms(x[key, : m["kv_rank"]], EPS) * W["dkv.norm"]) @ W["uk"].T).view(H, d)
    at = m["kv_rank"] + m["rot_dim"]
    q = x[query, at: at + H * (d + m["rot_dim"])].view(H, -1)
    q[:, :d] = exact(14.0 / m["scale"] * k / k.square().sum(-1, keepdim=True))
    q[:, d:] = 0


def run_latent(cases, m, schedule, dtype, device, bs=16):
    from miles_b200.ops import mixers as MX

    pages = U.Pages([len(c[0]) for c in cases], bs, device)
    lay = MX.LatentLayout(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"])
    W = {k: t.to(device=device, dtype=dtype) for k, t in cases[0][1].items()}
    freq = torch.tensor([m["rot"]["base"] ** (-2 * i / m["rot_dim"]) for i in range(m["rot_dim"] // 2)], dtype=torch.float64, device=device)
    cache = (50 * torch.randn(pages.num_blocks, bs, lay.pitch, generator=torch.Generator().manual_seed(9))).to(dtype).to(device)
    w_ukv, n_kv, n_q = torch.cat([W["uk"], W["uv"]]).contiguous(), m["kv_rank"] + m["rot_dim"], m["heads"] * (m["dim"] + m["rot_dim"])

    def fn(x, meta):
        x = whole(x, dtype, device)
        return MX.latent_attention(x[:, :n_kv], lay, cache, meta, freq=freq, magnitude=1.0, scale=m["scale"], window=0, sink=None, w_ukv=w_ukv,
                                   kv_norm=W["dkv.norm"], eps=EPS, q=x[:, n_kv: n_kv + n_q].contiguous(), gate=x[:, n_kv + n_q:])

    return U.run_pieces(pages, [c[0] for c in cases], schedule, fn)


def far_latents(device, dtype, m, T, pairs, tol, portions, bs=16):
    for query, key in pairs:
        case = latent_case(m, T, seed=query + key)
        point_latent(case, m, query, key)
        want = latent_want(case, m)
        for sizes in portions:
            got = run_latent([case], m, [[(0, n)] for n in U.sizes_for(T, sizes)], dtype, device, bs)[0]
            assert U.rel(got, want) < tol, (query, key, sizes, U.rel(got, want))
            assert U.rel(got[query:query + 1], want[query:query + 1]) < tol, (query, key, sizes)


# ---- row-wise mechanisms --------------------------------------------------------------------------------------------------------------------

def residuals(device, dtype, T, D, N, tol):
    """Residual sums with a factor: plain addends, normed ones, none; normed or as they are, alone and in front of a product."""
    from miles_b200.ops import mixers as MX

    g = torch.Generator().manual_seed(T + D)

    def rnd(*s, dt=dtype, k=1.0, mean=0.0):
        return (mean + k * torch.randn(*s, generator=g)).to(dt).to(device)

    x, y = rnd(T, D, dt=torch.float32), rnd(T, D)
    yn, nw, w = rnd(D, mean=1.0, k=0.2), rnd(D, mean=1.0, k=0.2), rnd(N, D, k=D ** -0.5)
    xd, yd = x.double(), y.double()
    for a, b, new in ((None, None, xd), (y, None, xd + 0.3 * yd), (y, yn, xd + 0.3 * plain.rms(yd, EPS) * yn.double())):
        for n in (nw, None):
            want = new if n is None else plain.rms(new, EPS) * n.double()
            with torch.no_grad():
                to = x.clone()
                h = MX.residual_norm(to, a, b, 0.3, n, EPS, dtype)
                assert U.rel(to, new) < 1e-6 and U.rel(h, want) < tol
                if MX.few_row_sum(x, (), w):
                    p, to = MX.residual_linear(x, a, b, 0.3, n, EPS, w)
                    assert U.rel(to, new) < 1e-6 and U.rel(p, want @ w.double().T) < 3 * tol
    with torch.no_grad():
        assert U.rel(MX.residual_norm(x.clone(), y, None, 0.3, nw, EPS, dtype, gain=0.5), 0.5 * plain.rms(xd + 0.3 * yd, EPS) * nw.double()) < tol


def activations(device, dtype, T, F, tol):
    from miles_b200.ops import mixers as MX

    g = torch.Generator().manual_seed(T)
    z = (4 * torch.randn(T, F, generator=g)).to(dtype)
    z[0, :3] = torch.tensor([0.0, -60.0, 40.0])
    for act in ((0.4, -1.3), (-2.0, 3.0)):
        a = torch.tensor(act).to(dtype)
        got = MX.xielu(z.to(device), a.to(device))
        want = plain.xielu(z.double(), a.double())
        assert float(((got.cpu().double() - want).abs() / (1 + want.abs())).max()) < tol
    table = exact(torch.randn(50, 3 * F, generator=g))
    tok = torch.randint(0, 50, (T,), generator=g)
    got = MX.gelu_times_rows(z.to(device), tok.int().to(device), table.to(device=device, dtype=dtype), F)
    want = plain.gelu_tanh(z.double()) * table[tok, F: 2 * F]
    assert float(((got.cpu().double() - want).abs() / (1 + want.abs())).max()) < tol
    x = 30 * torch.randn(T, F, generator=g)
    x[0, :3] = torch.tensor([0.0, -4000.0, 1e-4])
    got = MX.softcap_(x.clone().to(device), 7.0, exact=dtype == torch.float32)
    assert float((got.cpu().double() - 7.0 * torch.tanh(x.double() / 7.0)).abs().max()) < 5e-6


def greedy(cfg, W, prompt, n):
    """Greedy continuation by the plain model."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(plain.run(cfg, W, toks)[-1].argmax()))
    return toks[len(prompt):]
