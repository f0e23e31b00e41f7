"""Senadra on the CPU: configuration and names, the mechanisms' statements, cache / state / batching of the engine, generation."""
from __future__ import annotations

import json
import os

import pytest
import torch

import layered_utils as U
import plain_senadra as plain
import senadra_cases as cases
from miles_b200.models import designs, senadra
from miles_b200.models.config import ModelConfig, get_config
from miles_b200.models.convert import hf_state_to_ours, load_named_into_model, to_hf
from miles_b200.models.layered import AttentionSpec, DeltaSpec, LatentSpec, LayeredModel, XieluSpec
from miles_b200.models.qwen3 import build_model
from plain_senadra import attn, delta, latent, layer

F32 = dict(device="cpu", dtype=torch.float32)


@pytest.fixture(autouse=True)
def _few_threads():
    n = torch.get_num_threads()
    torch.set_num_threads(min(n, 4))
    yield
    torch.set_num_threads(n)


# ---- configuration, names, files ----------------------------------------------------------------------------------------

def test_config_round_trip_and_registry(tmp_path):
    for cfg in (cases.config_a(), cases.config_b(), cases.config_c()):
        c = ModelConfig.from_hf_config(cfg)
        assert c.family == "senadra" and c.block == "pre_norm" and not c.tie_embeddings
        assert senadra.from_config(c.to_hf_config()) == c
    c = ModelConfig.from_hf_config(cases.config_a())
    d, a, l = (c.layer_specs[i].mixer for i in range(3))
    assert isinstance(d, DeltaSpec) and (d.decay_rank, d.gate_rank, d.kv_heads) == (10, 7, 3)
    assert isinstance(a, AttentionSpec) and a.chunk == 20 and a.distance_bias and a.value_norm and a.gate and c.layer_specs[3].mixer.kv_from == 1
    assert isinstance(l, LatentSpec) and l.q_rank == 48 and l.gate and not l.sink and not l.window
    assert isinstance(c.layer_specs[0].mlp, XieluSpec) and c.layer_specs[2].mlp is None
    assert (c.residual_mult, c.logit_softcap, c.token_side, c.rms_eps) == (0.6, 12.0, 16, 1e-5)
    c.save(str(tmp_path))
    assert get_config(str(tmp_path)) == c
    assert isinstance(build_model(c, dtype=torch.float32), LayeredModel)
    assert get_config("senadra-tiny").family == "senadra" and designs.DESIGNS["senadra"].ARCHITECTURE == "Senadra"
    with pytest.raises(ValueError, match="unknown Senadra mixer"):
        senadra.from_config(dict(cases.config_a(), layers=[{"type": "x", "mixer": {}, "mlp": None}]))


def test_inner_sizes_come_from_the_tensors(tmp_path):
    """A configuration that does not name the inner sizes of the two-step projections, layers that differ in them."""
    from miles_b200.checkpoint.hf_io import save_safetensors

    cfg = cases.config_a()
    W = plain.make_weights(cfg)
    bare = json.loads(json.dumps(cfg))
    for l in bare["layers"]:
        l["mixer"].pop("decay_rank", None)
        l["mixer"].pop("gate_rank", None)
    (tmp_path / "config.json").write_text(json.dumps(bare))
    save_safetensors(str(tmp_path / "model.safetensors"), W)
    assert get_config(str(tmp_path)) == ModelConfig.from_hf_config(cfg)
    with pytest.raises(ValueError, match="decay_rank"):
        ModelConfig.from_hf_config(bare)


def test_a_layer_reads_only_an_earlier_layer_with_keys_of_its_own():
    for mixers in ([attn(kv_from=1), attn()], [attn(), attn(kv_heads=3), attn(kv_from=1)], [delta(), attn(kv_from=0)], [attn(), attn(kv_from=0), attn(kv_from=1)]):
        with pytest.raises(AssertionError, match="keys and values"):
            build_model(ModelConfig.from_hf_config(plain.make_config([layer(m, None) for m in mixers])), dtype=torch.float32)


def test_checkpoint_names_round_trip():
    cfg = cases.config_a()
    c, W = senadra.from_config(cfg), plain.make_weights(cfg)
    ours = hf_state_to_ours(W, c)
    model = build_model(c, dtype=torch.bfloat16)
    assert set(ours) == {n for n, _ in model.named_parameters()}
    for n, p in model.named_parameters():
        assert tuple(p.shape) == tuple(ours[n].shape) == designs.param_shapes(c)[n], n
    back = dict(kv for n, t in ours.items() for kv in to_hf(n, t, c))
    assert set(back) == set(W) and all(torch.equal(back[n], W[n]) for n in W)
    assert c.num_params() == sum(t.numel() for t in W.values())
    assert c.num_params(active_only=True) == c.num_params() - W["side.embed"].numel()


def test_weights_in_any_portions():
    """A weight stream may cut stacked projections and convolutions anywhere between tensors."""
    cfg = cases.config_a()
    c, W = senadra.from_config(cfg), plain.make_weights(cfg, 12)
    from miles_b200.parallel.state import ParallelState

    model = build_model(c, dtype=torch.float32)
    whole = hf_state_to_ours(W, c)
    for name, t in reversed(list(W.items())):
        load_named_into_model(model, [(name, t)], c, ParallelState.single())
    for n, p in model.named_parameters():
        assert torch.equal(p.data, whole[n].float()), n
    with pytest.raises(AssertionError, match="configuration says"):
        load_named_into_model(model, [("l0.mix.k.conv", torch.zeros(3, 4))], c, ParallelState.single())


def test_weights_from_disk(tmp_path):
    from miles_b200.checkpoint.hf_io import save_safetensors
    from miles_b200.engine.engine import Engine

    cfg = cases.config_b()
    W = plain.make_weights(cfg, 4)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_safetensors(str(tmp_path / "model.safetensors"), W)
    e = Engine(get_config(str(tmp_path)), num_blocks=8, max_running_requests=2, max_context_len=64, **F32)
    e.update_weights_from_disk(str(tmp_path))
    toks = U.tokens_for(cfg, 20)
    assert U.rel(U.feed_alone(e, toks, [20]), plain.run(cfg, W, toks)) < 1e-5
    del W["l2.mix.g2"]
    save_safetensors(str(tmp_path / "model.safetensors"), W)
    with pytest.raises(ValueError, match="lacks"):
        e.update_weights_from_disk(str(tmp_path))


def test_serving_build_of_a_configuration():
    from miles_b200.ops import build

    assert build.serve_kind(get_config("senadra-tiny")) == "attention_delta_latent_prep"
    assert build.serve_kind(ModelConfig.from_hf_config(plain.make_config([layer(delta())]))) == "delta"
    with open(os.path.join(build.CSRC, "bindings_mixers.cpp")) as f:
        text = f.read()
    for part, files in build.SERVE_PARTS.items():
        assert f"#ifdef MB_SERVE_{part.upper()}" in text and all(os.path.exists(os.path.join(build.CSRC, f)) for f in files), part


# ---- mechanisms ---------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("m", [delta(), delta(1, 1, 3, 5, 1, 2, 3), delta(4, 1, 8, 6, 5, 4, 1), delta(3, 3, 16, 8, 2)])
def test_delta_rule(m):
    case = cases.delta_case(m, 45, 1)
    want = cases.delta_want(case, m)
    for sizes in ([45], [1], [2], [20, 1, 9, 3]):
        assert U.rel(cases.run_delta([case], m, [[(0, n)] for n in U.sizes_for(45, sizes)], torch.float32, "cpu")[0], want) < 1e-5
    cases.remembered("cpu", torch.float32, m, 40, [(0, 39), (15, 16), (3, 30)], 1e-4, [[40], [16, 1, 7]])


def test_delta_rule_in_its_definition():
    """Unit keys that repeat: the second write replaces what the first one left, and the read-out sees its own token's write."""
    k = torch.zeros(3, 1, 4, dtype=torch.float64)
    k[:, 0, 1] = 1
    v = torch.tensor([[2.0, -1.0], [5.0, 3.0], [7.0, 7.0]], dtype=torch.float64)[:, None]
    o = plain.delta_rule(k, k, v, torch.zeros(3, 1, 4, dtype=torch.float64), torch.tensor([[1.0], [1.0], [0.5]], dtype=torch.float64))
    assert torch.allclose(o[:, 0], torch.tensor([[2.0, -1.0], [5.0, 3.0], [6.0, 5.0]], dtype=torch.float64))


def test_chunked_attention():
    for m in (attn(size=13), attn(heads=2, kv_heads=2, dim=5, vdim=3, size=16), attn(heads=4, kv_heads=1, dim=8, vdim=6, size=1), attn(size=100)):
        cases.pointed("cpu", torch.float32, m, 41, cases.edge_pairs(m["mask"]["size"], 41)[:12], 1e-4, [[41], [7, 2, 20], [1]])


def test_another_layers_keys_in_chunks_of_ones_own():
    m, other = attn(size=13), attn(heads=4, size=7, scale=0.7)
    case, mine = cases.attention_case(m, 40, 1), cases.attention_case(other, 40, 2)
    pages = U.Pages([40], 16)
    caches = cases.attention_caches(m, pages, torch.float32)
    U.run_pieces(pages, [case[0]], [[(0, 40)]], cases.attention_fn(m, case, caches, torch.float32, "cpu"))
    n = other["heads"] * other["dim"]
    q, gate = mine[0][:, :n], mine[0][:, -other["heads"] * other["vdim"]:]
    before = [c.clone() for c in caches]
    got = U.run_pieces(pages, [torch.cat([q, gate], -1)], [[(0, 25)], [(0, 15)]], cases.attention_fn(other, mine, caches, torch.float32, "cpu", writes=False))[0]
    k0 = m["heads"] * m["dim"]
    kv = case[0][:, k0: k0 + m["kv_heads"] * (m["dim"] + m["vdim"])]
    want = cases.attention_want((torch.cat([q, kv, gate], -1), mine[1]), other)
    assert U.rel(got, want) < 1e-5 and all(torch.equal(a, b) for a, b in zip(before, caches))


def test_latent_attention():
    for m in (latent(), latent(2, 5, 6, 3, 13, 11), latent(1, 16, 2, 8, 24, 8)):
        cases.far_latents("cpu", torch.float32, m, 41, [(40, 0), (40, 39), (17, 16), (16, 15), (0, 0), (20, 3)], 1e-4, [[41], [7, 2, 20], [1]])


@pytest.mark.parametrize("T,D,N", [(1, 12, 5), (7, 40, 9)])
def test_residual_sums(T, D, N):
    cases.residuals("cpu", torch.float32, T, D, N, 1e-5)


def test_activations():
    cases.activations("cpu", torch.float32, 9, 12, 1e-5)


# ---- the model in the engine -----------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name,T", [("a", 75), ("b", 61)])
def test_pieces_of_any_size(name, T):
    cfg = getattr(cases, f"config_{name}")()
    cases.sizes_for_all(F32, cfg, T, [[T], [T - 20] + [1] * 20, [2], [1, 30, 2, 3, 9, 17]], 3e-5)


def test_residual_after_every_layer():
    cfg = cases.config_a()
    W, toks, want = plain.make_weights(cfg, 7), U.tokens_for(cfg, 30, 1), []
    plain.run(cfg, W, toks, layers=want)
    e = U.engine_for(cfg, W, **F32)
    e.record_residual = got = []
    U.feed_alone(e, toks, [30])
    assert len(got) == len(want) == 5
    for a, b in zip(got, want):
        assert U.rel(a, b) < 1e-5


def test_mixed_batches_reuse_pages_and_slots():
    cases.mixed_batches(dict(F32, blocks=16, slots=3), cases.config_a(), [70, 41, 5, 66, 1, 30], 3e-5)


@pytest.mark.parametrize("kind", ["attention", "delta"])
def test_models_of_one_kind_of_layer(kind):
    """No states, or no pages: the engine keeps what the layers need."""
    mixers = [attn(), latent(), attn(kv_from=0)] if kind == "attention" else [delta(), delta(heads=2, kv_heads=2, conv=2)]
    cfg = plain.make_config([layer(m) for m in mixers])
    e = cases.sizes_for_all(F32, cfg, 40, [[40], [25] + [1] * 15], 3e-5, seed=2)
    assert len(e.kv.layers) == (2 if kind == "attention" else 0) and (e.states is None) == (kind == "attention")
    assert (e.prefix_cache is not None) == (kind == "attention")


def test_what_layers_keep():
    e = U.engine_for(cases.config_a(), plain.make_weights(cases.config_a()), **F32)
    assert set(e.kv.layers) == {1, 2} and set(e.states.layers) == {0, 4, (0, "conv")}      # one tap looks at nothing back


def test_without_optional_parts():
    """No soft cap, no token input."""
    cfg = cases.config_a()
    del cfg["logit_softcap"], cfg["token_side"]
    c = ModelConfig.from_hf_config(cfg)
    names = {n for n, _ in build_model(c, dtype=torch.float32).named_parameters()}
    assert not any("side" in n for n in names) and c.logit_softcap == 0.0 and senadra.from_config(c.to_hf_config()) == c


# ---- scheduler ------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("kw", [{}, {"chunked_prefill_size": 16}, {"chunked_prefill_size": 16, "mixed_batches": True},
                                {"share_prompt_kv": False, "mixed_batches": True}])
def test_greedy_generation(kw):
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 5)
    prompts = [U.tokens_for(cfg, n, n) for n in (37, 3, 20)]
    prompts.append(list(prompts[2]))                      # an identical prompt: shares pages, copies the states
    want = [cases.greedy(cfg, W, p, 10) for p in prompts[:3]]
    e = U.engine_for(cfg, W, slots=3, **F32, **kw)          # fewer slots than requests: a later one waits and joins while others run
    lengths = [10, 6, 10, 10]
    out = e.generate(prompts, [{"temperature": 0.0, "max_new_tokens": n} for n in lengths])
    assert [o["output_ids"] for o in out] == [w[:n] for w, n in zip(want + [want[2]], lengths)]
    if kw.get("mixed_batches"):
        assert e.stats.get("mixed_steps", 0) > 0


def test_retraction():
    """Too few pages for all: a request loses its pages and its states, starts again from its prompt and output, same tokens."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 6)
    prompts = [U.tokens_for(cfg, n, 40 + n) for n in (30, 29, 31)]
    want = [cases.greedy(cfg, W, p, 14) for p in prompts]
    e = U.engine_for(cfg, W, blocks=7, context=60, **F32)
    out = e.generate(prompts, {"temperature": 0.0, "max_new_tokens": 14})
    assert [o["output_ids"] for o in out] == want and e.stats["retractions"] > 0


def test_shared_prefixes_come_from_the_cache_of_attention_models():
    cfg = plain.make_config([layer(attn()), layer(latent()), layer(attn(kv_from=0))])
    W = plain.make_weights(cfg, 13)
    e = U.engine_for(cfg, W, **F32)
    prompt = U.tokens_for(cfg, 40, 6)
    for tail in ([], [3, 4, 5]):
        p = prompt + tail
        assert e.generate(p, {"temperature": 0.0, "max_new_tokens": 6})["output_ids"] == cases.greedy(cfg, W, p, 6)
    assert e.stats.get("prefix_cache_hit_tokens", 0) >= 32


def test_scoring_a_prompt():
    """The soft cap counts wherever rows meet the head."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 8)
    e = U.engine_for(cfg, W, **F32)
    toks = U.tokens_for(cfg, 25, 2)
    r = e.add_request(toks, {"temperature": 0.0, "max_new_tokens": 1}, logprob_start_len=0)
    while not r.done.is_set():
        e.step()
    lg = plain.run(cfg, W, toks)
    lp = torch.log_softmax(lg, -1)
    assert r.input_logprobs == pytest.approx([float(lp[i, toks[i + 1]]) for i in range(24)], abs=1e-4)
    assert float(lg.abs().max()) > 0.5 * cfg["logit_softcap"]      # the cap is felt
    got, entropy = e.model.log_probs(torch.randn(5, 64), torch.arange(5), 0.7, with_entropy=True)
    assert got.shape == entropy.shape == (5,) and bool((entropy > 0).all())


def test_memory_release_and_weight_update_keep_the_model():
    cfg = cases.config_a()
    W, W2 = plain.make_weights(cfg, 9), plain.make_weights(cfg, 10)
    e = U.engine_for(cfg, W, **F32)
    toks = U.tokens_for(cfg, 20, 3)
    e.release_memory_occupation()
    e.resume_memory_occupation()
    e.update_weights_from_tensor([kv for n, t in hf_state_to_ours(W2, e.cfg).items() for kv in to_hf(n, t, e.cfg)], weight_version=3)
    assert U.rel(U.feed_alone(e, toks, [12, 1, 7]), plain.run(cfg, W2, toks)) < 2e-5
