"""Nopelorn's kernels on the GPU against the plain model: bf16 (tensor-core kernels, decode graphs) and float32 (true 32-bit)."""
from __future__ import annotations

import pytest
import torch

import layered_utils as U
import nopelorn_cases as cases
import plain_nopelorn as plain

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
ENGINE_TOL = {torch.float32: 3e-5, torch.bfloat16: 0.08}      # whole models: bf16 products and activations in every layer
OP_TOL = {torch.float32: 2e-5, torch.bfloat16: 0.025}


def kw(dtype, **more):
    return dict(device="cuda:0", dtype=dtype, **more)


@pytest.fixture(autouse=True)
def _no_kernel_gave_up():
    yield
    from miles_b200.ops import cuda as K

    assert K.check_error_flag() == 0


# ---- whole models ----------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,T,bs", [("a", 90, 16), ("b", 61, 16), ("c", 230, 64)])
def test_pieces_of_any_size(name, T, bs, dtype):
    cfg = getattr(cases, f"config_{name}")()
    cases.sizes_for_all(kw(dtype, block_size=bs), cfg, T, [[T], [T - 40] + [1] * 40, [2], [1, 30, 2, 3, 9, 17, 64]], ENGINE_TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_reuse_pages_and_slots(dtype):
    cases.mixed_batches(kw(dtype, blocks=16), cases.config_a(), [70, 41, 5, 66, 1, 30], ENGINE_TOL[dtype])
    cases.mixed_batches(kw(dtype, blocks=10, block_size=64), cases.config_c(), [200, 150, 15, 90, 70], ENGINE_TOL[dtype])


def test_bf16_is_close_piece_by_piece():
    """The same request cut differently differs by much less than bf16 differs from the exact model."""
    cfg = cases.config_c()
    W, toks = plain.make_weights(cfg, 1), U.tokens_for(cfg, 150, 1)
    e = U.engine_for(cfg, W, **kw(torch.bfloat16, block_size=64))
    whole = U.feed_alone(e, toks, [150])
    for p in ([64, 3], [1, 2, 40]):
        assert U.rel(U.feed_alone(e, toks, U.sizes_for(150, p)), whole) < 0.06


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
    for p, o, n in zip(prompts, out, lengths):
        ids = o["output_ids"]
        assert len(ids) == n
        lg = plain.run(cfg, W, p + ids[:-1])[len(p) - 1:]
        lost = (lg.max(-1).values - lg.gather(1, torch.tensor(ids)[:, None])[:, 0]) / lg.std()
        assert float(lost.max()) < (1e-4 if dtype == torch.float32 else 0.25), lost
        lp = torch.log_softmax(lg, -1).gather(1, torch.tensor(ids)[:, None])[:, 0]
        got = torch.tensor([x[0] for x in o["meta_info"]["output_token_logprobs"]])
        assert float((lp - got).abs().max()) < (1e-3 if dtype == torch.float32 else 0.3)
    assert e.states.num_free == 3 and e.allocator.num_free == 40
    if dtype == torch.bfloat16:
        assert e.runner is not None and e.runner.graphs


def test_cache_sized_from_device_memory():
    """No block count given: pages from the memory budget, never more than the requests can fill; all preset layers run."""
    from miles_b200.engine.engine import Engine
    from miles_b200.models.config import get_config

    for layers in (4, 1):                        # 1: linear attention only, nothing cached per token
        e = Engine(get_config("nopelorn-tiny").with_(num_layers=layers), device="cuda:0", max_running_requests=3, max_context_len=256)
        assert e.kv.num_blocks == 3 * 5
        out = e.generate([[1, 2, 3] * 20, [7]], {"temperature": 0.0, "max_new_tokens": 40})
        assert [len(o["output_ids"]) for o in out] == [40, 40]


def test_eager_decode_without_graphs():
    cfg = cases.config_a()
    W, toks = plain.make_weights(cfg, 2), U.tokens_for(cfg, 60, 2)
    e = U.engine_for(cfg, W, use_cuda_graph=False, **kw(torch.bfloat16))
    assert U.rel(U.feed_alone(e, toks, [30] + [1] * 30), plain.run(cfg, W, toks)) < ENGINE_TOL[torch.bfloat16]


# ---- attention --------------------------------------------------------------------------------------------------------------

SPECS = {
    "one_atom": dict(heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=32, window=37),
    "two_atoms": dict(heads=20, dim=104, rot_dim=24, vdim=128, kv_rank=144, window=70),
    "mla": dict(heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=512, window=130),
    "narrow_values": dict(heads=33, dim=72, rot_dim=16, vdim=16, kv_rank=64, window=64),
    "odd": dict(heads=2, dim=9, rot_dim=6, vdim=5, kv_rank=19, window=21),
    "big_heads": dict(heads=2, dim=136, rot_dim=16, vdim=144, kv_rank=64, window=50),
    "big_rank": dict(heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=528, window=30),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SPECS))
def test_window_edges(name, dtype):
    m = plain.latent_spec(**SPECS[name])["mixer"]
    T = m["mask"]["size"] + 90
    # 1-token pieces take the decode form, ≤ 8 tokens the absorbed form, longer ones the expanded form
    cases.window_edges("cuda:0", dtype, m, T, OP_TOL[dtype], [[T], [T - 3, 1, 1, 1], [7, 2, 40]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["one_atom", "mla", "odd"])
def test_sink(name, dtype):
    cases.sink_counts("cuda:0", dtype, plain.latent_spec(**SPECS[name])["mixer"], 60, OP_TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_without_a_window(dtype):
    """No window: the last tokens of a long sequence point at its first, and at one in the middle of the pages."""
    m = dict(plain.latent_spec(heads=18, dim=40, rot_dim=16, vdim=24, kv_rank=48)["mixer"], mask=None)
    T = 700
    h, W = U.latent_case(m, T, 3)
    for key, query in ((0, T - 1), (333, T - 2), (64, 640)):
        U.point_at(h, W, m, cases.EPS, query, key, 20.0)
    want = plain.latent_attention(h, W, "x.", m, cases.EPS, plain.latent_of(h, W, "x.", m, cases.EPS))
    for sizes in ([T], [T - 70] + [1] * 70, [300, 5]):
        pages = U.Pages([T], 64, "cuda:0")
        cache = U.latent_cache(m, pages, dtype)
        got = U.run_pieces(pages, [h], [[(0, n)] for n in U.sizes_for(T, sizes)], U.latent_fn(m, W, cache, dtype, "cuda:0", cases.EPS))[0]
        assert U.rel(got, want) < OP_TOL[dtype], sizes


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_sequences_in_one_batch(dtype):
    m = plain.latent_spec(**SPECS["two_atoms"])["mixer"]
    lens = [300, 90, 17, 140, 9]
    schedule = [[(0, 200), (1, 9), (2, 3)], [(0, 5), (3, 130), (1, 64)], [(2, 1), (1, 1), (0, 1), (3, 1)], [(2, 1), (0, 70), (4, 9), (3, 8)],
                [(b, 100) for b in range(5)]]
    hs, ws = zip(*[U.latent_case(m, n, 1) for n in lens])
    hs = [U.latent_case(m, n, 10 + i)[0] for i, n in enumerate(lens)]
    W = ws[0]
    pages = U.Pages(lens, 16, "cuda:0")
    cache = U.latent_cache(m, pages, dtype)
    got = U.run_pieces(pages, hs, schedule, U.latent_fn(m, W, cache, dtype, "cuda:0", cases.EPS))
    for h, y in zip(hs, got):
        assert U.rel(y, plain.latent_attention(h, W, "x.", m, cases.EPS, plain.latent_of(h, W, "x.", m, cases.EPS))) < OP_TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_at_far_positions(dtype):
    """Scores depend on differences of positions only: a quarter of a million positions further on the answer is the same."""
    m = plain.latent_spec(heads=2, dim=16, rot_dim=32, vdim=16, kv_rank=32, window=25, factor=1.0)["mixer"]
    T, bs, shift = 60, 16, 16 * 16384
    h, W = U.latent_case(m, T, 4)
    want = plain.latent_attention(h, W, "x.", m, cases.EPS, plain.latent_of(h, W, "x.", m, cases.EPS))
    pages = U.Pages([T], bs, "cuda:0")
    cache = U.latent_cache(m, pages, dtype)
    fn = U.latent_fn(m, W, cache, dtype, "cuda:0", cases.EPS)

    def shifted(x, meta):
        meta.positions = meta.positions + shift
        meta.block_table = torch.cat([torch.zeros(len(meta.block_table), shift // bs, dtype=torch.int32, device="cuda"), meta.block_table], 1)
        if meta.ragged.seq_lens is not None:
            meta.ragged.seq_lens = [s + shift for s in meta.ragged.seq_lens]
        return fn(x, meta)

    # the window of the first shifted tokens reaches before the shift: compare where it does not
    got = U.run_pieces(pages, [h], [[(0, 40)], [(0, 5)], [(0, 1)], [(0, 14)]], shifted)[0]
    assert U.rel(got[25:], want[25:]) < max(OP_TOL[dtype], 5e-5)


# ---- linear attention ---------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dk,dv", [(2, 128, 128), (3, 40, 24), (1, 5, 3), (2, 16, 72), (2, 136, 8), (5, 64, 128)])
def test_linear_state(H, dk, dv, dtype):
    lengths = [330, 65, 9, 100]
    schedule = [[(0, 200), (1, 9), (2, 3)], [(0, 1), (1, 1), (2, 1)], [(0, 1), (3, 1)], [(3, 64), (1, 55), (2, 2), (0, 7)], [(0, 64), (3, 3)],
                [(b, 200) for b in range(4)]]
    cases.linear_state("cuda:0", dtype, H, dk, dv, lengths, schedule, OP_TOL[dtype], pull=(3, 329))


@pytest.mark.parametrize("decay", [[0.0, 1.0], [0.3, 0.9999]])
def test_linear_state_long_prompt_in_segments(decay):
    """Long enough to be cut into segments; a key at the start read at the end; decays of 0 and 1."""
    cases.linear_state("cuda:0", torch.bfloat16, 2, 128, 128, [2900, 700], [[(0, 2500), (1, 650)], [(0, 399), (1, 49)], [(0, 1), (1, 1)]],
                       OP_TOL[torch.bfloat16], decay=decay, pull=(5, 2899))


def test_segments_cover_every_token():
    from miles_b200.ops import mixers_cuda as MC

    for lens in ([9], [64, 65, 128], [2900, 700], [8192], [100] * 30):
        m = U.Pages(lens, 64, "cuda:0").meta([(b, 0, n) for b, n in enumerate(lens)])
        for H in (1, 2, 32):
            m.ragged.scratch.clear()
            segs, cu, multi = MC._segments(m, H)
            segs, cu = segs.tolist(), cu.tolist()
            at = 0
            for b, n in enumerate(lens):
                mine = segs[cu[b]:cu[b + 1]]
                assert [s[1] for s in mine] == [at] + [s[2] for s in mine[:-1]] and mine[-1][2] == at + n
                assert all(s[0] == b for s in mine) and [s[3] for s in mine] == [0] * (len(mine) - 1) + [1]
                assert all((s[2] - s[1]) % 64 == 0 for s in mine[:-1])
                at += n
            assert multi == (len(segs) > len(lens))


# ---- row-wise kernels -----------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,D", [(1, 64), (5, 37), (70, 2560), (3, 4104)])
def test_norms_embedding_and_activation(T, D, dtype):
    from miles_b200.ops import mixers as MX

    g = torch.Generator().manual_seed(T)

    def rnd(*s):
        return torch.randn(*s, generator=g).to(dtype).cuda()

    tol = 3e-6 if dtype == torch.float32 else 0.012
    x0, y, nw, ls, fw = torch.randn(T, D, generator=g).cuda(), rnd(T, D), rnd(D), rnd(D), rnd(D)
    want = x0.double() + plain.rms(y.double(), 1e-5) * nw.double() * ls.double()
    x, xb = MX.output_norm_residual(x0.clone(), y, nw, ls, 1e-5)
    assert x.dtype == torch.float32 and U.rel(x, want) < 3e-6 and U.rel(xb, want) < tol      # the residual is 32-bit in both
    x, xn = MX.output_norm_residual(x0.clone(), y, nw, ls, 1e-5, final_w=fw)
    assert U.rel(x, want) < 3e-6 and U.rel(xn, plain.rms(want, 1e-5) * fw.double()) < tol
    h = 3 * rnd(T, 2 * D)
    a, b = h.double().clamp(max=1.2)[:, :D], h.double()[:, D:].clamp(-1.2, 1.2)
    assert U.rel(MX.clamped_glu(h, 1.2, 1.702), a / (1 + torch.exp(-1.702 * a)) * (b + 1)) < tol
    gate = rnd(T, 3 * D)[:, D:2 * D]
    from miles_b200.ops import mixers_cuda as MC

    assert U.rel(MC.gated_norm(y, nw, gate, 1e-5), plain.rms(y.double(), 1e-5) * nw.double() / (1 + torch.exp(-gate.double()))) < tol
    V, B = 50, 11
    emb, tab = rnd(V, D), rnd(B + 1, D)
    tok = torch.randint(0, V, (T,), generator=g)
    prev = torch.cat([torch.tensor([-1]), tok[:-1]])
    got, _ = MX.bigram_embedding(tok.int().cuda(), prev.int().cuda(), emb, tab, (B, 10 ** 9 + 7, 3))
    rows = [B if p < 0 else (int(p) * (10 ** 9 + 7) + int(t) * 3) % B for p, t in zip(prev, tok)]
    assert torch.equal(got, emb[tok.cuda()].float() + tab[torch.tensor(rows).cuda()].float())


@pytest.mark.parametrize("M", [1, 3, 8, 16])
@pytest.mark.parametrize("K,N", [(64, 40), (2560, 300), (1056, 16)])
def test_output_norm_fused_into_a_projection(M, K, N):
    from miles_b200.ops import mixers_cuda as MC

    g = torch.Generator().manual_seed(M)
    x = torch.randn(M, K, generator=g).cuda()
    y, nw, ls, w = (torch.randn(*s, generator=g).bfloat16().cuda() for s in ((M, K), (K,), (K,), (N, K)))
    keep = x.clone()
    with torch.no_grad():
        out, x_new = MC.output_norm_linear(x, y, nw, ls, 1e-5, w)
    want = x.double() + plain.rms(y.double(), 1e-5) * nw.double() * ls.double()
    assert torch.equal(x, keep) and U.rel(x_new, want) < 3e-6
    assert U.rel(out, want @ w.double().T) < 0.012


@pytest.mark.parametrize("nk", [True, False])
@pytest.mark.parametrize("T,H,N,K", [(1, 6, 96, 64), (9, 3, 40, 24), (70, 8, 80, 512), (130, 40, 128, 128), (2, 2, 17, 9)])
def test_per_head_projection(T, H, N, K, nk):
    from miles_b200.ops import mixers_cuda as MC

    g = torch.Generator().manual_seed(T)
    x = torch.randn(T, H, K, generator=g).bfloat16().cuda()
    w = torch.randn(H, *((N, K) if nk else (K, N)), generator=g).bfloat16().cuda()
    want = torch.einsum("thk,hnk->thn" if nk else "thk,hkn->thn", x.double(), w.double())
    for fast in ([True, False] if N % 8 == 0 and K % 8 == 0 else [False]):
        y = torch.empty(T, H, N, dtype=torch.bfloat16, device="cuda")
        MC._head_linear(x, w, nk, y, fast)
        assert U.rel(y.flatten(1), want.flatten(1)) < 0.01


def test_odd_inner_sizes_in_the_dense_gemm():
    from miles_b200.ops import cuda as K

    g = torch.Generator().manual_seed(0)
    for M, N, Kd in ((5, 53, 37), (130, 131, 19), (40, 577, 100), (1, 7, 3), (5, 53, 64), (40, 577, 264), (20, 1001, 2048), (64, 333, 320)):
        a, b = torch.randn(M, Kd, generator=g).bfloat16().cuda(), torch.randn(N, Kd, generator=g).bfloat16().cuda()
        assert U.rel(K.gemm_nt(a, b), a.double() @ b.double().T) < 0.012
        assert U.rel(K.gemm_nt(a, b, out_dtype=torch.float32), a.double() @ b.double().T) < 1e-4
