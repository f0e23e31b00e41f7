"""Senadra's kernels on the GPU against the plain model: bf16 (tensor-core kernels, decode graphs) and float32 (true 32-bit)."""
from __future__ import annotations

import pytest
import torch

import layered_utils as U
import plain_senadra as plain
import senadra_cases as cases
from plain_senadra import attn, delta, latent, layer

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
ENGINE_TOL = {torch.float32: 3e-5, torch.bfloat16: 0.08}      # whole models: bf16 products and activations in every layer
OP_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.03}


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
@pytest.mark.parametrize("kind", ["attention", "delta"])
def test_models_of_one_kind_of_layer(kind, dtype):
    mixers = [attn(), latent(), attn(kv_from=0)] if kind == "attention" else [delta(), delta(heads=2, kv_heads=2, conv=2)]
    cases.sizes_for_all(kw(dtype), plain.make_config([layer(m) for m in mixers]), 40, [[40], [25] + [1] * 15], ENGINE_TOL[dtype], seed=2)


def test_residual_after_every_layer_in_32_bits():
    cfg = cases.config_c()
    W, toks, want = plain.make_weights(cfg, 7), U.tokens_for(cfg, 90, 1), []
    plain.run(cfg, W, toks, layers=want)
    e = U.engine_for(cfg, W, **kw(torch.float32))
    e.record_residual = got = []
    U.feed_alone(e, toks, [90])
    for a, b in zip(got, want, strict=True):
        assert U.rel(a, b) < 1e-5


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
    assert float(torch.cat(off).max()) < (1e-4 if dtype == torch.float32 else 0.2)
    if dtype == torch.bfloat16:
        assert e.runner is not None and e.runner.graphs


def test_cache_and_states_sized_from_device_memory():
    from miles_b200.engine.engine import Engine
    from miles_b200.models.config import get_config

    e = Engine(get_config("senadra-tiny"), device="cuda:0", max_running_requests=3, max_context_len=256)
    assert e.kv.num_blocks == 3 * 5 and len(e.kv.layers) == 2 and e.states.num_slots == 3
    out = e.generate([[1, 2, 3] * 20, [7]], {"temperature": 0.0, "max_new_tokens": 40})
    assert [len(o["output_ids"]) for o in out] == [40, 40]


def test_eager_decode_without_graphs():
    cfg = cases.config_a()
    W, toks = plain.make_weights(cfg, 2), U.tokens_for(cfg, 60, 2)
    e = U.engine_for(cfg, W, use_cuda_graph=False, **kw(torch.bfloat16))
    cases.close(U.feed_alone(e, toks, [30] + [1] * 30), plain.run(cfg, W, toks), ENGINE_TOL[torch.bfloat16])


# ---- delta rule -----------------------------------------------------------------------------------------------------------------

DELTAS = {
    "full": delta(2, 2, 128, 128, 4, 32, 16),
    "shared_keys": delta(6, 2, 64, 64, 4, 16, 24),
    "narrow_keys": delta(3, 1, 16, 128, 3, 8, 8),
    "narrow_values": delta(2, 2, 104, 24, 2, 16, 8),
    "one_and_a_bit": delta(3, 3, 72, 40, 5, 24, 8),
    "smallest_tiles": delta(2, 1, 8, 8, 1, 3, 5),
    "large": delta(2, 1, 160, 144, 4, 8, 8),                  # token by token
    "odd": delta(3, 3, 9, 7, 6, 5, 3),
    "many_taps": delta(2, 2, 16, 16, 20, 8, 8),
    "off_the_grid": delta(1, 1, 9, 7, 2, 32, 64),             # inner rows of whole steps that start between 16-byte boundaries
}


def same_weights(cs):
    return [(c[0], cs[0][1]) for c in cs]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("forget", [False, True])
@pytest.mark.parametrize("name", sorted(DELTAS))
def test_delta_rule(name, forget, dtype):
    m = DELTAS[name]
    cs = same_weights([cases.delta_case(m, n, i, forget) for i, n in enumerate([200, 90, 17])])
    schedules = [[[(0, 200), (1, 90), (2, 17)]], [[(0, 70), (1, 1), (2, 9)], [(0, 1), (1, 64), (2, 2)], [(0, 65), (1, 9), (2, 1)]] + [[(0, 64), (1, 30), (2, 30)]],
                 [[(0, 150)], [(1, 80)], [(2, 1)]] + [[(0, 1), (1, 1), (2, 1)]] * 12 + [[(0, 2), (2, 3)]] * 2 + [[(0, 40)]]]
    want = [cases.delta_want(c, m) for c in cs]
    for s in schedules:
        for y, w in zip(cases.run_delta(cs, m, s, dtype, "cuda:0"), want):
            assert U.rel(y, w[: len(y)]) < OP_TOL[dtype], (s, U.rel(y, w[: len(y)]))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["full", "shared_keys", "one_and_a_bit", "large"])
def test_what_a_state_remembers(name, dtype):
    """Over blocks of 16 and chunks of 64 tokens, pieces and decode steps."""
    T = 200
    pairs = [(0, T - 1), (15, 16), (0, 47), (63, 64), (64, 127), (127, 128), (10, 150), (T - 2, T - 1)]
    cases.remembered("cuda:0", dtype, DELTAS[name], T, pairs, OP_TOL[dtype], [[T], [64, 1, 63, 2], [T - 50] + [1] * 50])


def test_rounds_of_chunks(monkeypatch):
    """Little room for what the first kernel leaves: every piece goes through in several rounds, its state through its slot."""
    from miles_b200.ops import mixers_cuda as MC

    m = DELTAS["shared_keys"]
    cs = same_weights([cases.delta_case(m, n, i) for i, n in enumerate((430, 90, 9))])
    want = [cases.delta_want(c, m) for c in cs]
    monkeypatch.setattr(MC, "DELTA_SCRATCH", 3 * m["heads"] * MC.C.delta_chunk_bytes(m["dim"], m["vdim"]))
    for s in ([[(0, 430), (1, 90), (2, 9)]], [[(0, 70), (1, 3)], [(0, 300), (1, 87), (2, 9)], [(0, 60)]]):
        for y, w in zip(cases.run_delta(cs, m, s, torch.bfloat16, "cuda:0"), want):
            assert U.rel(y, w) < OP_TOL[torch.bfloat16]


@pytest.mark.parametrize("warps", [2, 4, 8])
def test_slices_of_value_columns(warps, monkeypatch):
    from miles_b200.ops import mixers_cuda as MC

    monkeypatch.setattr(MC, "scan_warps", lambda *a: warps)
    for name in ("full", "narrow_values", "one_and_a_bit", "smallest_tiles"):
        m = DELTAS[name]
        cs = same_weights([cases.delta_case(m, n, i) for i, n in enumerate((150, 64))])
        for y, c in zip(cases.run_delta(cs, m, [[(0, 80), (1, 64)], [(0, 70)]], torch.bfloat16, "cuda:0"), cs):
            assert U.rel(y, cases.delta_want(c, m)) < OP_TOL[torch.bfloat16], name


def test_chunks_keep_more_than_16_bits():
    """The chunked form against the token-by-token one on the same rounded inputs: what is left are the two-part operands."""
    from miles_b200.ops import mixers_cuda as MC

    m = dict(DELTAS["full"])
    case = cases.delta_case(m, 192, 3)
    args = [[case], m, [[(0, 192)]], torch.bfloat16, "cuda:0"]
    chunked = cases.run_delta(*args)[0]
    one = cases.run_delta([case], m, [[(0, 8)]] * 24, torch.bfloat16, "cuda:0")[0]      # short pieces take the recurrence itself
    assert MC.scan_warps(2, 128) in (2, 4, 8) and U.rel(chunked, one) < 4e-3       # outputs are bf16: two roundings apart


@pytest.mark.parametrize("rows", [1, 40, 200])
def test_many_rows_of_a_decode_step(rows):
    m = delta(8, 4, 72, 32, 4, 16, 8)
    cs = same_weights([cases.delta_case(m, 11, i) for i in range(rows)])
    want = [cases.delta_want(c, m) for c in cs[:7]]
    for dtype in DTYPES:
        out = cases.run_delta(cs, m, [[(b, 9) for b in range(rows)]] + [[(b, 1) for b in range(rows)]] * 2, dtype, "cuda:0")
        for y, w in zip(out, want):
            assert U.rel(y, w) < OP_TOL[dtype]
    pages = U.Pages([1, 1], 16, "cuda:0")                     # a padding row takes no part
    meta = pages.meta([(0, 0, 1), (1, 0, 1)], decode_form=True)
    meta.state_slots[1] = -1
    y = cases.delta_fn(m, cs[0], pages, torch.bfloat16, "cuda:0")(cs[0][0][:2].cuda(), meta)
    assert bool((y[1] == 0).all()) and U.rel(y[:1], cases.delta_want((cs[0][0][:1], cs[0][1]), m)) < OP_TOL[torch.bfloat16]


# ---- chunked attention --------------------------------------------------------------------------------------------------------------

ATTNS = {
    "small": attn(4, 2, 24, 40, size=37),
    "full": attn(8, 2, 128, 128, size=64),
    "long_chunks": attn(4, 1, 64, 64, size=150),
    "one_chunk": attn(4, 4, 48, 72, size=1000),
    "group_of_12": attn(12, 1, 40, 128, size=90),
    "short_chunks": attn(2, 1, 104, 16, size=5),
    "single_tokens": attn(2, 2, 16, 16, size=1),
    "odd": attn(3, 1, 9, 5, size=33),
    "large": attn(2, 1, 136, 144, size=50),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ATTNS))
def test_chunked_attention(name, dtype):
    m = ATTNS[name]
    cs = same_weights([cases.attention_case(m, n, i) for i, n in enumerate([200, 90, 17])])
    for bs in (16, 64, 24):
        for s in ([[(0, 200), (1, 90), (2, 17)]], [[(0, 70), (1, 1), (2, 9)], [(0, 1), (1, 64), (2, 2)], [(0, 65), (1, 9), (2, 1)], [(0, 64), (1, 30), (2, 30)]],
                  [[(0, 150)], [(1, 80)], [(2, 1)]] + [[(0, 1), (1, 1), (2, 1)]] * 12):
            for y, c in zip(cases.run_attention(cs, m, s, dtype, "cuda:0", bs), cs):
                assert U.rel(y, cases.attention_want(c, m)[: len(y)]) < OP_TOL[dtype], (bs, s)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["small", "full", "long_chunks", "short_chunks", "odd", "large"])
def test_edges_of_chunks(name, dtype):
    m, T = ATTNS[name], 160
    pairs = cases.edge_pairs(m["mask"]["size"], T)[:14]
    cases.pointed("cuda:0", dtype, m, T, pairs, 1e-4 if dtype == torch.float32 else OP_TOL[dtype], [[T], [64, 1, 63, 2], [T - 100] + [1] * 100], 64)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 70])
def test_decode_over_long_chunks(rows, dtype):
    """Several splits of the keys, one and many rows."""
    m = attn(8, 2, 64, 128, size=700)
    cs = same_weights([cases.attention_case(m, 690 if i < 2 else 40, i) for i in range(rows)])
    out = cases.run_attention(cs, m, [[(b, 685 if b < 2 else 35) for b in range(rows)]] + [[(b, 1) for b in range(rows)]] * 5, dtype, "cuda:0", 64)
    for y, c in list(zip(out, cs))[:4]:
        assert U.rel(y, cases.attention_want(c, m)) < OP_TOL[dtype]


# ---- latent attention ---------------------------------------------------------------------------------------------------------------

LATENTS = {
    "small": latent(3, 24, 16, 40, 56),
    "full": latent(4, 128, 64, 128, 512),
    "many_heads": latent(34, 32, 16, 24, 64),
    "odd": latent(2, 5, 6, 3, 13),
    "wide_values": latent(2, 72, 32, 136, 96),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(LATENTS))
def test_latent_attention(name, dtype):
    m = LATENTS[name]
    cs = same_weights([cases.latent_case(m, n, i) for i, n in enumerate([150, 70, 12])])
    for bs in (16, 64):
        for s in ([[(0, 150), (1, 70), (2, 12)]], [[(0, 70), (1, 1)], [(0, 1), (1, 64), (2, 2)], [(0, 79), (1, 5), (2, 10)]], [[(0, 140), (1, 60), (2, 3)]] + [[(0, 1), (1, 1), (2, 1)]] * 9):
            for y, c in zip(cases.run_latent(cs, m, s, dtype, "cuda:0", bs), cs):
                assert U.rel(y, cases.latent_want(c, m)[: len(y)]) < OP_TOL[dtype], (bs, s)
    cases.far_latents("cuda:0", dtype, m, 150, [(149, 0), (149, 64), (64, 63), (0, 0), (130, 15)], 1e-4 if dtype == torch.float32 else OP_TOL[dtype],
                      [[150], [64, 1, 63, 2], [100] + [1] * 50], 64)


# ---- row-wise mechanisms ----------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,D,N", [(1, 64, 40), (3, 2560, 96), (4, 96, 7), (40, 1024, 64), (9, 37, 21), (300, 200, 72)])
def test_residual_sums(T, D, N, dtype):
    cases.residuals("cuda:0", dtype, T, D, N, 1e-5 if dtype == torch.float32 else 0.004)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,F", [(1, 40), (30, 72), (7, 13), (200, 1000)])
def test_activations(T, F, dtype):
    cases.activations("cuda:0", dtype, T, F, 2e-6 if dtype == torch.float32 else 0.006)
