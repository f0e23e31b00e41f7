"""Vozirax's kernels on the GPU against the plain model: bf16 (tensor-core kernels, decode graphs) and float32 (true 32-bit)."""
from __future__ import annotations

import pytest
import torch

import layered_utils as U
import plain_vozirax as plain
import vozirax_cases as cases
from plain_vozirax import attn, ff, layer, moe, ssm

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
ENGINE_TOL = {torch.float32: 3e-5, torch.bfloat16: 0.08}      # whole models: bf16 products and activations in every layer
OP_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.04}


def kw(dtype, **more):
    return dict(device="cuda:0", dtype=dtype, **more)


@pytest.fixture(autouse=True)
def _no_kernel_gave_up():
    yield
    from miles_b200.ops import cuda as K

    assert K.check_error_flag() == 0


# ---- whole models ----------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,T,bs", [("a", 90, 16), ("b", 61, 16), ("c", 230, 64), ("c", 150, 24)])
def test_pieces_of_any_size(name, T, bs, dtype):
    cfg = getattr(cases, f"config_{name}")()
    cases.sizes_for_all(kw(dtype, block_size=bs), cfg, T, [[T], [T - 40] + [1] * 40, [2], [1, 30, 2, 3, 9, 17, 64]], ENGINE_TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_reuse_pages_and_slots(dtype):
    cases.mixed_batches(kw(dtype, blocks=16, slots=3), cases.config_a(), [70, 41, 5, 66, 1, 30], ENGINE_TOL[dtype])
    cases.mixed_batches(kw(dtype, blocks=10, block_size=64), cases.config_c(), [200, 150, 15, 90, 70], ENGINE_TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    cases.sizes_for_all(kw(dtype), cases.config_a(), 260, [[20] + [1] * 240], ENGINE_TOL[dtype], seed=4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "ssm"])
def test_models_of_one_kind_of_layer(kind, dtype):
    mixers = [attn(), attn(kv_from=0)] if kind == "attention" else [ssm(), ssm(heads=2, groups=1, norm_groups=2)]
    cfg = plain.make_config([layer(mixers[0], ff()), layer(mixers[1], moe())])
    cases.sizes_for_all(kw(dtype), cfg, 40, [[40], [25] + [1] * 15], ENGINE_TOL[dtype], seed=2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("opts", [{}, {"chunked_prefill_size": 32, "mixed_batches": True}])
def test_generation(dtype, opts):
    """Greedy generation through the scheduler, long enough for several round trips of the decode graphs; every choice is the plain
    model's, or within rounding of it."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 5, apart=dtype == torch.bfloat16)
    prompts = [U.tokens_for(cfg, n, n) for n in (37, 3, 20)]
    prompts.append(list(prompts[2]))
    lengths = [70, 25, 40, 40]
    e = U.engine_for(cfg, W, slots=3, **kw(dtype, blocks=40), **opts)
    out = e.generate(prompts, [{"temperature": 0.0, "max_new_tokens": n} for n in lengths])
    off = []
    for p, o, n in zip(prompts, out, lengths):
        ids = o["output_ids"]
        assert len(ids) == n
        lg = plain.run(cfg, W, p + ids[:-1])[len(p) - 1:]
        off.append((lg.max(-1).values - lg.gather(1, torch.tensor(ids)[:, None])[:, 0]) / lg.std())
    assert float(torch.cat(off).max()) < (1e-4 if dtype == torch.float32 else 0.2)
    if dtype == torch.bfloat16:
        assert e.runner is not None and e.runner.graphs


def test_cache_and_states_sized_from_device_memory():
    from miles_b200.engine.engine import Engine
    from miles_b200.models.config import get_config

    e = Engine(get_config("vozirax-tiny"), device="cuda:0", max_running_requests=3, max_context_len=256)
    assert e.kv.num_blocks == 3 * 5 and len(e.kv.layers) == 1 and e.states.num_slots == 3
    out = e.generate([[1, 2, 3] * 20, [7]], {"temperature": 0.0, "max_new_tokens": 40})
    assert [len(o["output_ids"]) for o in out] == [40, 40]


def test_eager_decode_without_graphs():
    cfg = cases.config_a()
    W, toks = plain.make_weights(cfg, 2, apart=True), U.tokens_for(cfg, 60, 2)
    e = U.engine_for(cfg, W, use_cuda_graph=False, **kw(torch.bfloat16))
    cases.close(U.feed_alone(e, toks, [30] + [1] * 30), plain.run(cfg, W, toks), ENGINE_TOL[torch.bfloat16])


# ---- state-space mixer ------------------------------------------------------------------------------------------------------

SSMS = {
    "pairs": dict(heads=4, vdim=64, state=128, groups=2, taps=4),             # two heads per tile, whole tiles
    "narrow_pairs": dict(heads=8, vdim=16, state=24, groups=2, taps=3),
    "pairs_48": dict(heads=6, vdim=48, state=88, groups=1, taps=2),
    "odd_group": dict(heads=6, vdim=32, state=64, groups=2, taps=4),          # three heads per group: one per tile
    "wide": dict(heads=2, vdim=128, state=128, groups=2, taps=4),
    "one_and_a_bit": dict(heads=3, vdim=72, state=40, groups=1, taps=5),
    "no_look_back": dict(heads=2, vdim=8, state=8, groups=1, taps=1),
    "large_state": dict(heads=2, vdim=24, state=160, groups=1, taps=4),       # token by token
    "odd": dict(heads=3, vdim=7, state=9, groups=3, taps=6),
    "many_taps": dict(heads=2, vdim=16, state=16, groups=1, taps=20),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SSMS))
def test_state_space(name, dtype):
    m = ssm(**SSMS[name])
    lens = [200, 90, 17]
    cs = [cases.ssm_case(m, n, i) for i, n in enumerate(lens)]
    cs = [(c[0], cs[0][1]) for c in cs]
    schedules = [[[(0, 200), (1, 90), (2, 17)]], [[(0, 70), (1, 1), (2, 9)], [(0, 1), (1, 64), (2, 2)], [(0, 65), (1, 9), (2, 1)]] + [[(0, 64), (1, 30), (2, 30)]],
                 [[(0, 150)], [(1, 80)], [(2, 1)]] + [[(0, 1), (1, 1), (2, 1)]] * 12 + [[(0, 2), (2, 3)]] * 2 + [[(0, 40)]]]
    for s in schedules:
        for c, y in zip(cs, cases.run_ssm(cs, m, s, dtype, "cuda:0")):
            assert U.rel(y, cases.ssm_want((c[0][: len(y)], c[1]), m)) < OP_TOL[dtype], s


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["pairs", "odd_group", "one_and_a_bit", "large_state"])
def test_what_a_state_remembers(name, dtype):
    """Over chunks of 64 tokens, segments of chunks, pieces and decode steps."""
    m = ssm(**SSMS[name])
    T = 300
    pairs = [(0, T - 1), (63, 64), (64, 127), (127, 128), (10, 250), (255, 256), (T - 2, T - 1)]
    cases.remembered("cuda:0", dtype, m, T, pairs, OP_TOL[dtype], [[T], [64, 1, 63, 2], [T - 50] + [1] * 50])


@pytest.mark.parametrize("size", [64, 128, 192])
def test_segments(size, monkeypatch):
    """A long prompt cut into segments of any number of chunks, from nothing and from a state."""
    from miles_b200.ops import mixers_cuda as MC

    monkeypatch.setattr(MC, "_segment_cost", lambda chunks, c, H, sms=148: abs(c - size // 64) + 0.1)
    for name in ("pairs", "wide"):
        m = ssm(**SSMS[name])
        cs = [cases.ssm_case(m, n, i) for i, n in enumerate((530, 140))]
        cs = [(c[0], cs[0][1]) for c in cs]
        for s in ([[(0, 530), (1, 140)]], [[(0, 70), (1, 3)], [(0, 400), (1, 137)], [(0, 60)]]):
            for c, y in zip(cs, cases.run_ssm(cs, m, s, torch.bfloat16, "cuda:0")):
                assert U.rel(y, cases.ssm_want(c, m)) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("rows", [1, 40, 200])
def test_many_rows_of_a_decode_step(rows):
    """One and two heads per CTA of the decode kernel; a padding row takes no part."""
    m = ssm(heads=8, vdim=32, state=72, groups=2, taps=4)
    cs = [cases.ssm_case(m, 11, i) for i in range(rows)]
    cs = [(c[0], cs[0][1]) for c in cs]
    want = [cases.ssm_want(c, m) for c in cs[:7]]
    for dtype in DTYPES:
        out = cases.run_ssm(cs, m, [[(b, 9) for b in range(rows)]] + [[(b, 1) for b in range(rows)]] * 2, dtype, "cuda:0")
        for y, w in zip(out, want):
            assert U.rel(y, w) < OP_TOL[dtype]
    pages = U.Pages([1, 1], 16, "cuda:0")
    meta = pages.meta([(0, 0, 1), (1, 0, 1)], decode_form=True)
    meta.state_slots[1] = -1
    y = cases.ssm_fn(m, cs[0], pages, torch.bfloat16, "cuda:0")(cs[0][0][:2].cuda(), meta)
    assert bool((y[1] == 0).all()) and U.rel(y[:1], cases.ssm_want((cs[0][0][:1], cs[0][1]), m)) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,C,parts,N", [(1, 64, 1, 40), (4, 4096, 1, 96), (16, 96, 1, 8), (40, 1024, 1, 64), (3, 96, 4, 24), (70, 90, 6, 10), (5, 12000, 2, 16)])
def test_norm_in_parts(M, C, parts, N, dtype):
    from miles_b200.ops import mixers as MX

    g = torch.Generator().manual_seed(M)
    x, w, wo = (torch.randn(*s, generator=g).to(dtype).cuda() for s in ((M, C), (C,), (N, C)))
    with torch.no_grad():
        y = MX.part_norm_linear(x, w, parts, 1e-5, wo)
    want = (plain.rms(x.double().unflatten(-1, (parts, -1)), 1e-5).flatten(-2) * w.double()) @ wo.double().T
    assert U.rel(y, want) < (1e-5 if dtype == torch.float32 else 0.012)


# ---- differential attention -----------------------------------------------------------------------------------------------------

ATTNS = {
    "one_atom": dict(heads=4, kv_heads=2, dim=24, vdim=40),
    "two_atoms": dict(heads=6, kv_heads=2, dim=56, vdim=120),
    "full": dict(heads=4, kv_heads=1, dim=64, vdim=128),                 # eight rows of a key head
    "sixteen_rows": dict(heads=16, kv_heads=2, dim=64, vdim=128),
    "uneven_rows": dict(heads=20, kv_heads=2, dim=32, vdim=64),          # twenty rows: sixteen and four
    "narrow_values": dict(heads=3, kv_heads=3, dim=64, vdim=16),
    "wide_values": dict(heads=12, kv_heads=1, dim=16, vdim=128),
    "odd": dict(heads=3, kv_heads=1, dim=9, vdim=5),
    "big_maps": dict(heads=2, kv_heads=1, dim=72, vdim=144),
    "bigger_maps": dict(heads=2, kv_heads=2, dim=264, vdim=24),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ATTNS))
def test_pointed_queries(name, dtype):
    m = cases.sharp(**ATTNS[name], every=20)
    T = 150
    pairs = [(T - 1, 0, 77), (T - 1, 64, 63), (100, 15, 16), (64, 64, 0), (63, 62, 63), (T - 3, T - 2, 5), (0, 0, 0), (40, 39, 41)]
    # 1-token pieces take the decode form, ≤ 8 tokens the decode kernel row by row, longer ones the prefill kernel
    cases.pointed("cuda:0", dtype, m, T, pairs, OP_TOL[dtype], [[T], [T - 3, 1, 1, 1], [7, 2, 40]])


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys(dtype):
    """The last tokens of a long sequence point at its first, and at ones among hundreds."""
    m = cases.sharp(heads=4, kv_heads=2, dim=32, vdim=64, every=100, coef=0.2)
    T = 700
    case = cases.attention_case(m, T, 3)
    for query, key, key2 in ((T - 1, 0, 600), (T - 2, 333, 1), (640, 64, 63), (T - 5, 8, 500), (T - 6, 127, 128)):
        cases.point_at(case, m, query, key, key2)
    want = cases.attention_want(case, m)
    for sizes in ([T], [T - 70] + [1] * 70, [300, 5]):
        got = cases.run_attention([case], m, [[(0, n)] for n in U.sizes_for(T, sizes)], dtype, "cuda:0", 64)[0]
        assert U.rel(got, want) < OP_TOL[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bs", [8, 12, 24, 64, 128])
def test_unequal_sequences_on_pages_of_any_size(bs, dtype):
    m = cases.sharp(**ATTNS["full"], every=50)
    lens = [300, 90, 17, 140, 9]
    schedule = [[(0, 200), (1, 9), (2, 3)], [(0, 5), (3, 130), (1, 64)], [(2, 1), (1, 1), (0, 1), (3, 1)], [(2, 1), (0, 70), (4, 9), (3, 8)],
                [(b, 100) for b in range(5)]]
    cs = [cases.attention_case(m, n, 10 + i) for i, n in enumerate(lens)]
    cs = [(c[0], cs[0][1]) for c in cs]
    for query, key in ((299, 0), (bs, bs - 1), (150, min(2 * bs, 149)), (202, bs)):
        cases.point_at(cs[0], m, query, key, query - 1)
    for c, y in zip(cs, cases.run_attention(cs, m, schedule, dtype, "cuda:0", bs)):
        assert U.rel(y, cases.attention_want(c, m)) < OP_TOL[dtype]


@pytest.mark.parametrize("name", ["full", "sixteen_rows", "uneven_rows", "narrow_values"])
@pytest.mark.parametrize("splits", [1, 2, 5, 8])
def test_any_number_of_splits(splits, name, monkeypatch):
    from miles_b200.ops import mixers_cuda as MC

    monkeypatch.setattr(MC, "window_splits", lambda *a: splits)
    m = cases.sharp(**ATTNS[name])
    case = cases.attention_case(m, 420, 1)
    got = cases.run_attention([case], m, [[(0, 380)]] + [[(0, 1)]] * 20 + [[(0, 8)]] * 3, torch.bfloat16, "cuda:0", 64)[0]
    assert U.rel(got, cases.attention_want(case, m)) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_and_values_of_another_layer(dtype):
    """Queries and gates of its own, nothing written."""
    m = cases.sharp(**ATTNS["one_atom"])
    n = cases.sharp(**ATTNS["one_atom"], diff=0.7, every=6)
    own, other = cases.attention_case(m, 60, 1), cases.attention_case(n, 60, 2)
    pages = U.Pages([60], 16, "cuda:0")
    caches = cases.attention_caches(m, pages, dtype)
    write, read = (cases.attention_fn(s, c, caches, dtype, "cuda:0", writes=w) for s, c, w in ((m, own, True), (n, other, False)))
    q, _, _, gate = cases.attention_split(other[0], n)
    rows = torch.cat([own[0], q, gate], 1)
    at, first = own[0].shape[1], []

    def both(x, meta):
        first.append(write(x[:, :at], meta).cpu())
        keep = [c.clone() for c in caches]
        y = read(x[:, at:].contiguous(), meta)
        assert all(torch.equal(a, b) for a, b in zip(caches, keep))
        return y

    got = U.run_pieces(pages, [rows], [[(0, 30)], [(0, 5)], [(0, 1)], [(0, 24)]], both)[0]
    mixed = torch.cat([q, *cases.attention_split(own[0], m)[1:3], gate], 1)
    want = cases.attention_want((mixed, dict(other[1], **{"k.norm": own[1]["k.norm"]})), n)
    assert U.rel(got, want) < OP_TOL[dtype] and U.rel(torch.cat(first), cases.attention_want(own, m)) < OP_TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_equal_maps(dtype):
    """Both maps the same: o = (1 − λ) a before its norm; what is left of the subtraction is still 32-bit."""
    m = cases.sharp(heads=4, kv_heads=2, dim=32, vdim=64, diff=0.8)
    case = cases.attention_case(m, 120, 6)
    q, k, _, _ = (t.clone() for t in cases.attention_split(case[0], m))
    q, k = (t.unflatten(-1, (-1, 2, 32)) for t in (q, k))
    q[:, :, 1], k[:, :, 1] = q[:, :, 0], k[:, :, 0]
    case[0][:, : 4 * 64], case[0][:, 4 * 64: 6 * 64] = q.flatten(1), k.flatten(1)
    want = cases.attention_want(case, m)
    for sizes in ([120], [100] + [1] * 20):
        assert U.rel(cases.run_attention([case], m, [[(0, n)] for n in sizes], dtype, "cuda:0", 64)[0], want) < OP_TOL[dtype]


# ---- embedding, choice of experts, experts, sums ----------------------------------------------------------------------------------

@pytest.mark.parametrize("width", [37, 64, 2048])
def test_position_vectors(width):
    cases.embedding("cuda:0", torch.float32, width, 1e-6)
    cases.embedding("cuda:0", torch.bfloat16, width, 2e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,k,count,keep", cases.CHOICES)
def test_choice_of_experts(T, E, k, count, keep, dtype):
    """Beside every kernel that may do it: attention preparation, convolution, decode step."""
    ms, ma = ssm(heads=2, vdim=8, state=8, groups=1, taps=3), attn(heads=2, kv_heads=1, dim=8, vdim=8)
    sc, ac = cases.ssm_case(ms, T), cases.attention_case(ma, T)
    pages = U.Pages([T], 16, "cuda:0")
    decode = U.Pages([1] * T, 16, "cuda:0")

    def beside_attention(a):
        cases.attention_fn(ma, ac, cases.attention_caches(ma, pages, dtype), dtype, "cuda:0", a)(ac[0].cuda(), pages.meta([(0, 0, T)]))

    def beside_convolution(a):
        cases.ssm_fn(ms, sc, pages, dtype, "cuda:0", a)(sc[0].cuda(), pages.meta([(0, 0, T)]))

    def beside_step(a):
        cases.ssm_fn(ms, sc, decode, dtype, "cuda:0", a)(sc[0].cuda(), decode.meta([(b, 0, 1) for b in range(T)], decode_form=True))

    for run in (beside_attention, beside_convolution, beside_step):
        cases.choice("cuda:0", dtype, T, E, k, count, keep, run)


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_activation_on_the_way(dtype):
    from miles_b200.ops import mixers as MX

    ms, ma = ssm(heads=2, vdim=8, state=8, groups=1, taps=3), attn(heads=2, kv_heads=1, dim=8, vdim=8)
    for T, F in ((9, 24), (30, 13)):
        sc, ac = cases.ssm_case(ms, T), cases.attention_case(ma, T)
        pages, g = U.Pages([T], 16, "cuda:0"), torch.randn(T, 2 * F, generator=torch.Generator().manual_seed(T)).to(dtype).cuda()
        want = torch.nn.functional.silu(g.double()[:, :F]) * g.double()[:, F:]
        for fn, x in ((cases.attention_fn(ma, ac, cases.attention_caches(ma, pages, dtype), dtype, "cuda:0"), ac[0]),
                      (cases.ssm_fn(ms, sc, pages, dtype, "cuda:0"), sc[0])):
            a = MX.Aside(glu_in=g, glu_out=torch.empty(T, F, dtype=dtype, device="cuda"), limit=float("inf"), alpha=1.0, shift=0.0)
            (cases.attention_fn(ma, ac, cases.attention_caches(ma, pages, dtype), dtype, "cuda:0", a) if x is ac[0] else
             cases.ssm_fn(ms, sc, pages, dtype, "cuda:0", a))(x.cuda(), pages.meta([(0, 0, T)]))
            assert U.rel(a.glu_out, want) < (1e-5 if dtype == torch.float32 else 0.01)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,k,D,F", [(1, 6, 2, 64, 32), (8, 16, 8, 256, 96), (3, 1, 1, 32, 32),       # matrix-vector kernels
                                       (40, 12, 3, 192, 96), (130, 5, 5, 64, 40), (20, 200, 2, 128, 64),   # small grouped tiles
                                       (700, 6, 2, 256, 128), (400, 2, 2, 72, 24),                         # 128-row tiles
                                       (9, 5, 2, 37, 11), (33, 3, 1, 64, 12)])                             # any size
def test_experts(T, E, k, D, F, dtype):
    cases.experts("cuda:0", dtype, T, E, k, D, F, 1e-5 if dtype == torch.float32 else 0.025, skew=T in (40, 700))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,D", [(1, 64), (5, 37), (70, 2048), (3, 13000)])
def test_sums_and_norms(T, D, dtype):
    cases.sums("cuda:0", dtype, T, D, 3e-6 if dtype == torch.float32 else 0.012)


@pytest.mark.parametrize("M", [1, 3, 8, 16])
@pytest.mark.parametrize("K,N,E,routes", [(64, 41, 5, True), (2048, 300, 128, True), (1056, 16, 90, False), (64, 24, 0, False)])
def test_sum_two_norms_and_products_in_one_kernel(M, K, N, E, routes):
    from miles_b200.ops import mixers as MX
    from miles_b200.ops import mixers_cuda as MC

    g = torch.Generator().manual_seed(M)
    x = torch.randn(M, K, generator=g).cuda()
    y1, y2, s1, s2, n1, n2, w, r = (torch.randn(*s, generator=g).bfloat16().cuda() for s in ((M, K), (M, K), (K,), (K,), (K,), (K,), (N, K), (max(E, 1), K)))
    keep = x.clone()
    with torch.no_grad():
        for adds in ([], [MX.Addend(y1, scale=s1)], [MX.Addend(y1, scale=s1), MX.Addend(y2, scale=s2)]):
            proj, second, h2, x_new = MC.sum_two_norms_linear(x, adds, n1, w, n2 if E else None, r if E else None, 1e-5, 1.0, routes)
            want = x.double() + sum(a.y.double() * a.scale.double() for a in adds)
            n = plain.rms(want, 1e-5)
            assert torch.equal(x, keep) and U.rel(x_new, want) < 1e-6 and proj.dtype == torch.bfloat16
            assert U.rel(proj, (n * (1 + n1.double())) @ w.double().T) < 0.012
            if E:
                lg = (n * (1 + n2.double())) @ r.double().T
                assert second.dtype == (torch.float32 if routes else torch.bfloat16)
                assert float((second.double() - lg).abs().max() / lg.square().mean().sqrt()) < (0.02 if routes else 0.03)
            if routes:
                assert U.rel(h2, n * (1 + n2.double())) < 0.012
