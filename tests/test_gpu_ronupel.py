"""Ronupel's kernels on the GPU against the plain model: bf16 (tensor-core kernels, decode graphs) and float32 (true 32-bit)."""
from __future__ import annotations

import pytest
import torch

import layered_utils as U
import plain_ronupel as plain
import ronupel_cases as cases

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
ENGINE_TOL = {torch.float32: 3e-5, torch.bfloat16: 0.08}      # whole models: bf16 products and activations in every layer
OP_TOL = {torch.float32: 2e-5, torch.bfloat16: 0.04}


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
def test_mixed_batches_reuse_pages(dtype):
    cases.mixed_batches(kw(dtype, blocks=16), cases.config_a(), [70, 41, 5, 66, 1, 30], ENGINE_TOL[dtype])
    cases.mixed_batches(kw(dtype, blocks=10, block_size=64), cases.config_c(), [200, 150, 15, 90, 70], ENGINE_TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """Far past every window and several pages, the kept tokens still in sight."""
    cfg = cases.config_a()
    cases.sizes_for_all(kw(dtype), cfg, 260, [[20] + [1] * 240], ENGINE_TOL[dtype], seed=4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("loop", [None, (0, 4, 2), (2, 4, 3)])
def test_loops(loop, dtype):
    cfg = dict(cases.config_a(), loop=dict(zip(("start", "stop", "times"), loop)) if loop else None)
    cases.sizes_for_all(kw(dtype), cfg, 50, [[50], [20] + [1] * 30], ENGINE_TOL[dtype], seed=2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("opts", [{}, {"chunked_prefill_size": 32, "mixed_batches": True}])
def test_generation(dtype, opts):
    """Greedy generation through the scheduler, long enough for several round trips of the decode graphs; every choice is the plain
    model's, or within rounding of it."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 5)
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
    off = torch.cat(off)
    # (in 16 bits a token may choose another, equally good expert: a few choices may lose more)
    assert float(off.max()) < (1e-4 if dtype == torch.float32 else 1.0) and float(off.quantile(0.97)) < (1e-4 if dtype == torch.float32 else 0.25)
    if dtype == torch.bfloat16:
        assert e.runner is not None and e.runner.graphs


def test_routing_recorded_in_the_decode_graphs():
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 8)
    e = U.engine_for(cfg, W, **kw(torch.bfloat16))
    out = e.generate([U.tokens_for(cfg, 20, 2)], {"temperature": 0.0, "max_new_tokens": 30}, return_routed_experts=True)[0]
    toks = U.tokens_for(cfg, 20, 2) + out["output_ids"]
    from miles_b200.types import decode_routed_experts

    got = out["meta_info"]["routed_experts"]
    got = torch.as_tensor(got if not isinstance(got, (str, bytes)) else decode_routed_experts(got, 50, 5, 3))[:49]
    assert got.shape == (49, 5, 3)
    h = plain.rms(W["embed"].double()[torch.tensor(toks[:49])], W["l0.norm1"].double(), 1e-5)
    idx, _ = plain.choose(h @ W["l0.mlp.router"].double().T + W["l0.mlp.router.b"].double(), 2)
    assert (got[:, 0, :2].sort(-1).values == idx.sort(-1).values).float().mean() > 0.97 and bool((got[:, 0, 2] == -1).all())


def test_cache_sized_from_device_memory():
    from miles_b200.engine.engine import Engine
    from miles_b200.models.config import get_config

    e = Engine(get_config("ronupel-tiny"), device="cuda:0", max_running_requests=3, max_context_len=256)
    assert e.kv.num_blocks == 3 * 5 and len(e.kv.layers) == 6
    out = e.generate([[1, 2, 3] * 20, [7]], {"temperature": 0.0, "max_new_tokens": 40})
    assert [len(o["output_ids"]) for o in out] == [40, 40]


def test_eager_decode_without_graphs():
    cfg = cases.config_a()
    W, toks = plain.make_weights(cfg, 2), U.tokens_for(cfg, 60, 2)
    e = U.engine_for(cfg, W, use_cuda_graph=False, **kw(torch.bfloat16))
    cases.close(U.feed_alone(e, toks, [30] + [1] * 30), plain.run(cfg, W, toks), ENGINE_TOL[torch.bfloat16])


# ---- attention --------------------------------------------------------------------------------------------------------------

SPECS = {
    "one_atom": dict(heads=4, kv_heads=2, dim=24, vdim=40, rot=8, window=37, keep=9),
    "two_atoms": dict(heads=6, kv_heads=2, dim=104, vdim=128, rot=64, window=70, keep=65),
    "full_heads": dict(heads=8, kv_heads=2, dim=128, vdim=128, rot=128, window=130, keep=4),
    "narrow_values": dict(heads=5, kv_heads=5, dim=128, vdim=16, rot=32, window=64, keep=64),
    "wide_values": dict(heads=7, kv_heads=1, dim=16, vdim=128, rot=16, window=40, keep=1),
    "many_heads": dict(heads=40, kv_heads=2, dim=64, vdim=64, rot=64, window=50, keep=20),      # three chunks of 8 per key head
    "keeps_a_lot": dict(heads=2, kv_heads=1, dim=32, vdim=32, rot=16, window=9, keep=100),
    "odd": dict(heads=3, kv_heads=1, dim=9, vdim=5, rot=6, window=21, keep=7),
    "big_heads": dict(heads=2, kv_heads=1, dim=136, vdim=144, rot=72, window=50, keep=3),
}


def spec(name, **more):
    m = dict(SPECS[name], **more)
    return plain.mixer_spec(**m, scale=3.0 / m["dim"] ** 0.5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SPECS))
def test_edges(name, dtype):
    m = spec(name)
    T = m["mask"]["size"] + m["mask"]["keep_first"] + 70
    # 1-token pieces take the decode form, ≤ 8 tokens the decode kernel row by row, longer ones the prefill kernel
    cases.edges("cuda:0", dtype, m, T, OP_TOL[dtype], [[T], [T - 3, 1, 1, 1], [7, 2, 40]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bs", [8, 12, 24, 32, 64, 128])
def test_page_sizes(bs, dtype):
    """Pages of one or several boxes, pages larger than a key tile, and a size the prefill kernel leaves to the any-size one."""
    m = spec("two_atoms")
    lens = [200, 90]
    cs = [cases.attention_case(m, n, 3 + i) for i, n in enumerate(lens)]
    cs = [(c[0], *cs[0][1:]) for c in cs]
    for key, query in ((0, 199), (bs - 1, 150), (min(2 * bs, 110), min(2 * bs, 110) + 69), (64, 133)):
        cases.point_at(cs[0], m, query, key)
    got = cases.run_attention(cs, m, [[(0, 90), (1, 33)], [(0, 3), (1, 1)], [(1, 56), (0, 7)], [(0, 1)], [(0, 99)]], dtype, "cuda:0", bs)
    for c, y in zip(cs, got):
        assert U.rel(y, cases.attention_want(c, m)) < OP_TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["one_atom", "full_heads", "odd"])
def test_sinks(name, dtype):
    m = plain.mixer_spec(**SPECS[name], scale=SPECS[name]["dim"] ** -0.5)
    cases.sinks("cuda:0", dtype, m, 60, OP_TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [0, 600])
def test_far_keys(window, dtype):
    """No window, or a wide one: the last tokens of a long sequence point at its first, and at ones among hundreds."""
    m = spec("one_atom", window=window)
    T = 700
    case = cases.attention_case(m, T, 3)
    for key, query in ((0, T - 1), (333, T - 2), (64, 640), (8, T - 5), (9, T - 6), (T - 10 - 599, T - 10), (T - 11 - 600, T - 11)):
        cases.point_at(case, m, query, key)
    want = cases.attention_want(case, m)
    for sizes in ([T], [T - 70] + [1] * 70, [300, 5]):
        got = cases.run_attention([case], m, [[(0, n)] for n in U.sizes_for(T, sizes)], dtype, "cuda:0", 64)[0]
        assert U.rel(got, want) < OP_TOL[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_sequences_in_one_batch(dtype):
    m = spec("two_atoms")
    lens = [300, 90, 17, 140, 9]
    schedule = [[(0, 200), (1, 9), (2, 3)], [(0, 5), (3, 130), (1, 64)], [(2, 1), (1, 1), (0, 1), (3, 1)], [(2, 1), (0, 70), (4, 9), (3, 8)],
                [(b, 100) for b in range(5)]]
    cs = [cases.attention_case(m, n, 10 + i) for i, n in enumerate(lens)]
    cs = [(c[0], *cs[0][1:]) for c in cs]
    for c, y in zip(cs, cases.run_attention(cs, m, schedule, dtype, "cuda:0")):
        assert U.rel(y, cases.attention_want(c, m)) < OP_TOL[dtype]


@pytest.mark.parametrize("splits", range(1, 9))
def test_any_number_of_splits(splits, monkeypatch):
    from miles_b200.ops import mixers_cuda as MC

    monkeypatch.setattr(MC, "window_splits", lambda *a: splits)
    m = spec("full_heads", window=300, keep=50)
    case = cases.attention_case(m, 420, 1)
    got = cases.run_attention([case], m, [[(0, 380)]] + [[(0, 1)]] * 20 + [[(0, 8)]] * 3, torch.bfloat16, "cuda:0", 64)[0]
    assert U.rel(got, cases.attention_want(case, m)) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_at_far_positions(dtype):
    """Scores depend on differences of positions only: a quarter of a million positions further on the answer is the same."""
    m = spec("one_atom", window=25, keep=0, rot=24, factor=1.0)
    T, bs, shift = 60, 16, 16 * 16384
    case = cases.attention_case(m, T, 4)
    pages = U.Pages([T], bs, "cuda:0")
    fn = cases.attention_fn(m, case, cases.attention_caches(m, pages, dtype), dtype, "cuda:0")

    def shifted(x, meta):
        meta.positions = meta.positions + shift
        meta.block_table = torch.cat([torch.zeros(len(meta.block_table), shift // bs, dtype=torch.int32, device="cuda"), meta.block_table], 1)
        if meta.ragged.seq_lens is not None:
            meta.ragged.seq_lens = [s + shift for s in meta.ragged.seq_lens]
        return fn(x, meta)

    # the window of the first shifted tokens reaches before the shift: compare where it does not
    got = U.run_pieces(pages, [case[0]], [[(0, 40)], [(0, 5)], [(0, 1)], [(0, 14)]], shifted)[0]
    assert U.rel(got[25:], cases.attention_want(case, m)[25:]) < max(OP_TOL[dtype], 5e-5)


# ---- experts, sums, projections ---------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,k,D,F", [(1, 6, 2, 64, 32), (8, 16, 8, 256, 96), (3, 1, 1, 32, 32),       # matrix-vector kernels
                                       (40, 12, 3, 192, 96), (130, 5, 5, 64, 40), (20, 200, 2, 128, 64),   # small grouped tiles
                                       (700, 6, 2, 256, 128), (400, 2, 2, 72, 24),                         # 128-row tiles
                                       (9, 5, 2, 37, 11), (33, 3, 1, 64, 12)])                             # any size
def test_experts(T, E, k, D, F, dtype):
    cases.experts("cuda:0", dtype, T, E, k, D, F, 1e-5 if dtype == torch.float32 else 0.02, skew=T in (40, 700))


@pytest.mark.parametrize("T,E,k", [(1, 1, 1), (5, 12, 2), (70, 128, 8), (9, 300, 40), (3, 33, 33)])
def test_choice_of_experts(T, E, k):
    from miles_b200.ops import mixers as MX

    m = plain.mixer_spec(heads=2, kv_heads=1, dim=8, vdim=8, rot=8)
    z = torch.randn(T, E, generator=torch.Generator().manual_seed(E))
    z[0, : E // 2 + 1] = 2.0                           # equal logits: the lower index
    if E > 1:
        z[-1, 0] = -float("inf")
    for dtype in DTYPES:
        aside = MX.Aside(logits=z.cuda(), top=k)
        g = torch.randn(T, 64, generator=torch.Generator().manual_seed(1)).to(dtype).cuda()
        aside.glu_in, aside.glu_out, aside.limit, aside.alpha = g[:, 8:40], torch.zeros(T, 24, dtype=dtype, device="cuda")[:, 4:20], 0.7, 1.702
        pages = U.Pages([T], 16, "cuda:0")
        case = cases.attention_case(m, T, 0)
        lay = MX.AttentionLayout(2, 1, 8, 8, 0, 4, 0)
        MX.windowed_attention(case[0].to(dtype).cuda(), lay, *cases.attention_caches(m, pages, dtype), pages.meta([(0, 0, T)]),
                              torch.empty(T, 16, dtype=dtype, device="cuda"), freq=torch.zeros(0, dtype=torch.float64, device="cuda"), magnitude=1.0,
                              scale=0.3, sink=None, q_norm=None, k_norm=None, eps=1e-5, aside=aside)
        idx, w = plain.choose(z.double(), k)
        assert torch.equal(aside.index.cpu().long(), idx) and torch.allclose(aside.weights.cpu().double(), w, atol=1e-6 if dtype == torch.float32 else 1e-5)
        gd = g.double().cpu()
        assert U.rel(aside.glu_out, plain.glu(gd[:, 8:24], gd[:, 24:40], 0.7)) < (1e-5 if dtype == torch.float32 else 0.01)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,D", [(1, 64), (5, 37), (70, 2048), (3, 13000)])
def test_sum_and_norm(T, D, dtype):
    from miles_b200.ops import mixers as MX

    g = torch.Generator().manual_seed(T)

    def rnd(*s, dt=dtype):
        return torch.randn(*s, generator=g).to(dt).cuda()

    x, extra, nw, a, b, rows = rnd(T, D, dt=torch.float32), rnd(T, D, dt=torch.float32), rnd(D), rnd(T, D), rnd(T, D), rnd(3 * T, D)
    w, dst = torch.rand(T, 3, generator=g).cuda(), torch.randperm(3 * T, generator=g).int().cuda()
    dst[0] = -1                                        # a choice that took no part
    gathered = (w.double()[..., None] * torch.where(dst[:, None] >= 0, rows.double()[dst.long()], 0.0).view(T, 3, D)).sum(1)
    keep = x.clone()
    for adds, ex, want in (([], None, x.double()), ([MX.Addend(a)], None, x.double() + a.double()),
                           ([MX.Addend(a), MX.Addend(b)], extra, x.double() + a.double() + b.double() + extra.double()),
                           ([MX.Addend(a), MX.Addend(rows, w, dst)], None, x.double() + a.double() + gathered)):
        to = torch.empty_like(x)
        h = MX.sum_norm(x, to, adds, ex, nw, 1e-5)
        assert torch.equal(x, keep) and U.rel(to, want) < 1e-6      # the residual is 32-bit in both
        assert h.dtype == dtype and U.rel(h, plain.rms(want, nw.double(), 1e-5)) < (3e-6 if dtype == torch.float32 else 0.012)


@pytest.mark.parametrize("M", [1, 3, 8, 16])
@pytest.mark.parametrize("K,N,E", [(64, 40, 5), (2048, 300, 128), (1056, 16, 1)])
def test_sum_norm_and_two_products_in_one_kernel(M, K, N, E):
    from miles_b200.ops import mixers as MX
    from miles_b200.ops import mixers_cuda as MC

    g = torch.Generator().manual_seed(M)
    x, extra = (torch.randn(M, K, generator=g).cuda() for _ in range(2))
    y1, y2, nw, w, r, b = (torch.randn(*s, generator=g).bfloat16().cuda() for s in ((M, K), (M, K), (K,), (N, K), (E, K), (E,)))
    keep = x.clone()
    with torch.no_grad():
        for adds, ex in (([], None), ([MX.Addend(y1)], None), ([MX.Addend(y1), MX.Addend(y2)], extra)):
            h, proj, logits, x_new = MC.sum_norm_linear(x, adds, ex, nw, 1e-5, w, r, b, True)
            want = x.double() + sum(a.y.double() for a in adds) + (ex.double() if ex is not None else 0)
            n = plain.rms(want, nw.double(), 1e-5)
            assert torch.equal(x, keep) and U.rel(x_new, want) < 1e-6 and U.rel(h, n) < 0.012
            assert proj.dtype == torch.bfloat16 and U.rel(proj, n @ w.double().T) < 0.012
            lg = n @ r.double().T + b.double()
            assert logits.dtype == torch.float32 and float((logits.double() - lg).abs().max() / lg.square().mean().sqrt()) < 0.02
        # the products alone: logits are exact sums of the rounded rows
        proj, logits = MC.projections(h, w, r, b)
        lg = h.double() @ r.double().T + b.double()
        assert U.rel(proj, h.double() @ w.double().T) < 0.012 and float((logits.double() - lg).abs().max() / lg.square().mean().sqrt()) < 1e-5


@pytest.mark.parametrize("T", [40, 300])
def test_router_logits_of_many_rows(T):
    from miles_b200.ops import mixers_cuda as MC

    g = torch.Generator().manual_seed(T)
    h, w, r, b = (torch.randn(*s, generator=g).bfloat16().cuda() for s in ((T, 192), (80, 192), (13, 192), (13,)))
    with torch.no_grad():
        proj, logits = MC.projections(h, w, r, b)
    lg = h.double() @ r.double().T + b.double()
    assert logits.dtype == torch.float32 and float((logits.double() - lg).abs().max() / lg.square().mean().sqrt()) < 1e-5
    assert U.rel(proj, h.double() @ w.double().T) < 0.012
