"""Vozirax on the CPU: configuration and names, the mechanisms' statements, cache / state / batching of the engine, generation."""
from __future__ import annotations

import json
import os

import pytest
import torch

import layered_utils as U
import plain_vozirax as plain
import vozirax_cases as cases
from miles_b200.models import designs, vozirax
from miles_b200.models.config import ModelConfig, get_config
from miles_b200.models.convert import hf_state_to_ours, load_named_into_model, to_hf
from miles_b200.models.layered import DifferentialSpec, LayeredModel, MoeSpec, ReluSquareSpec, SsmSpec
from miles_b200.models.qwen3 import build_model
from miles_b200.ops import mixers as MX
from plain_vozirax import attn, ff, layer, moe, ssm

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
        assert c.family == "vozirax" and c.block == "two_norms" and not c.tie_embeddings
        assert vozirax.from_config(c.to_hf_config()) == c
    c = ModelConfig.from_hf_config(cases.config_a())
    a, s, f = c.layer_specs[1].mixer, c.layer_specs[0].mixer, c.layer_specs[1].mlp
    assert isinstance(a, DifferentialSpec) and a.temperature.every == 9 and c.layer_specs[3].mixer.kv_from == 1
    assert isinstance(s, SsmSpec) and s.norm_groups == 3 and c.layer_specs[2].mlp is None and c.layer_specs[3].mixer.temperature is None
    assert isinstance(f, MoeSpec) and isinstance(f.expert, ReluSquareSpec) and f.routing == MX.Routing(4, 2, 1.7)
    assert c.layer_specs[3].mlp.routing.groups == 1 and c.num_experts == 8 and c.moe_topk == 3 and c.num_moe_layers == 3
    c.save(str(tmp_path))
    assert get_config(str(tmp_path)) == c
    assert isinstance(build_model(c, dtype=torch.float32), LayeredModel)
    assert get_config("vozirax-tiny").family == "vozirax" and designs.DESIGNS["vozirax"].ARCHITECTURE == "Vozirax"
    with pytest.raises(ValueError, match="unknown Vozirax mixer"):
        vozirax.from_config(dict(cases.config_a(), layers=[{"type": "x", "mixer": {}, "mlp": None}]))


def test_a_layer_reads_only_an_earlier_layer_with_keys_of_its_own():
    for mixers in ([attn(kv_from=1), attn()], [attn(), attn(kv_heads=2), attn(kv_from=1)], [ssm(), attn(kv_from=0)]):
        cfg = plain.make_config([layer(m, None) for m in mixers])
        if mixers[-1].get("kv_from") == 1:
            cfg["layers"][2]["mixer"]["kv_heads"] = 3
        with pytest.raises(AssertionError, match="keys and values"):
            build_model(ModelConfig.from_hf_config(cfg), dtype=torch.float32)


def test_checkpoint_names_round_trip():
    cfg = cases.config_a()
    c, W = vozirax.from_config(cfg), plain.make_weights(cfg)
    ours = hf_state_to_ours(W, c)
    model = build_model(c, dtype=torch.bfloat16)
    assert set(ours) == {n for n, _ in model.named_parameters()}
    for n, p in model.named_parameters():
        assert tuple(p.shape) == tuple(ours[n].shape) == designs.param_shapes(c)[n], n
    back = dict(kv for n, t in ours.items() for kv in to_hf(n, t, c))
    assert set(back) == set(W) and all(torch.equal(back[n], W[n]) for n in W)
    assert c.num_params() == sum(t.numel() for t in W.values())
    unused = 64 * 2 * ((8 - 3) * 40 + (5 - 2) * 24 + (8 - 2) * 40)
    assert c.num_params(active_only=True) == c.num_params() - unused


def test_weights_in_any_portions():
    """A weight stream may cut stacked projections, vectors and experts anywhere between tensors."""
    cfg = cases.config_a()
    c, W = vozirax.from_config(cfg), plain.make_weights(cfg, 12)
    from miles_b200.parallel.state import ParallelState

    model = build_model(c, dtype=torch.float32)
    whole = hf_state_to_ours(W, c)
    for name, t in reversed(list(W.items())):
        load_named_into_model(model, [(name, t)], c, ParallelState.single())
    for n, p in model.named_parameters():
        assert torch.equal(p.data, whole[n].float()), n
    with pytest.raises(AssertionError, match="configuration says"):
        load_named_into_model(model, [("l1.mix.lk2", torch.zeros(3))], c, ParallelState.single())


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
    del W["l0.mix.lk1"]
    save_safetensors(str(tmp_path / "model.safetensors"), W)
    with pytest.raises(ValueError, match="lacks"):
        e.update_weights_from_disk(str(tmp_path))


def test_serving_build_of_a_configuration():
    from miles_b200.ops import build

    assert build.serve_kind(get_config("vozirax-tiny")) == "attention_differential_experts_ssm"
    for part, files in build.SERVE_PARTS.items():       # the part with experts registers their bindings, every other one its mixers'
        registered = "bindings_more.cpp" if "bindings_moe.cpp" in files else "bindings_mixers.cpp"
        with open(os.path.join(build.CSRC, registered)) as f:
            assert f"MB_SERVE_{part.upper()})" in f.read() or registered == "bindings_mixers.cpp", part


# ---- mechanisms ---------------------------------------------------------------------------------------------------------------

def test_position_vectors():
    for width in (16, 37):
        cases.embedding("cpu", torch.float32, width, 1e-6)
        assert torch.allclose(plain.place_vectors(9, width)[5, 2:4], torch.tensor([torch.sin(torch.tensor(5.0).double() * 10000.0 ** (-2 / width)),
                                                                                  torch.cos(torch.tensor(5.0).double() * 10000.0 ** (-2 / width))]))


@pytest.mark.parametrize("m", [ssm(), ssm(heads=1, vdim=3, state=5, groups=1, taps=1), ssm(heads=4, vdim=8, state=6, groups=4, taps=5)])
def test_state_space(m):
    case = cases.ssm_case(m, 45, 1)
    want = cases.ssm_want(case, m)
    for sizes in ([45], [1], [2], [20, 1, 9, 3]):
        assert U.rel(cases.run_ssm([case], m, [[(0, n)] for n in U.sizes_for(45, sizes)], torch.float32, "cpu")[0], want) < 1e-5
    cases.remembered("cpu", torch.float32, m, 40, [(0, 39), (15, 16), (3, 30)], 1e-4, [[40], [16, 1, 7]])


def test_step_sizes_are_not_clamped():
    z = torch.tensor([-80.0, -20.0, 0.0, 3.0, 90.0], dtype=torch.float64)
    got = plain.step_sizes(z, torch.zeros(5, dtype=torch.float64))
    assert float(got[0]) > 0 and float(got[4]) == pytest.approx(90.0) and torch.allclose(got, torch.nn.functional.softplus(z, threshold=1000))


def test_differential_attention():
    for m in (cases.sharp(), cases.sharp(heads=2, kv_heads=2, dim=5, vdim=3, coef=None), cases.sharp(heads=4, kv_heads=1, dim=8, vdim=6, every=7)):
        pairs = [(39, 0, 20), (39, 38, 39), (17, 16, 15), (16, 15, 0), (0, 0, 0), (20, 21, 3)]
        cases.pointed("cpu", torch.float32, m, 41, pairs, 1e-4, [[41], [7, 2, 20], [1]])


def test_temperature_steps():
    """The factor changes at the position that completes `every` tokens, the first one included."""
    t = plain.temperature(20, {"coef": 0.5, "every": 4})
    assert [round(float(v), 6) for v in t[:5]] == [1.0, 1.0, 1.0, round(1 + 0.5 * 0.6931471805599453, 6), round(1 + 0.5 * 0.6931471805599453, 6)]
    m = cases.sharp(coef=0.9, every=4)
    case = cases.attention_case(m, 20, 2)
    assert U.rel(cases.run_attention([case], m, [[(0, 20)]], torch.float32, "cpu")[0], cases.attention_want(case, m)) < 1e-5
    off = cases.attention_want(case, dict(m, q_temp={"coef": 0.9, "every": 5}))
    assert float(U.row_errors(off, cases.attention_want(case, m))[3]) > 0.01


@pytest.mark.parametrize("T,E,k,count,keep", cases.CHOICES)
def test_choice_of_experts(T, E, k, count, keep):
    from miles_b200.ops import mixers_reference as ref

    cases.choice("cpu", torch.float32, T, E, k, count, keep, ref.aside)


@pytest.mark.parametrize("T,E,k,D,F", [(9, 5, 2, 16, 12), (1, 1, 1, 7, 5), (30, 3, 3, 8, 10)])
def test_experts(T, E, k, D, F):
    cases.experts("cpu", torch.float32, T, E, k, D, F, 1e-5)


def test_sums_and_norms():
    cases.sums("cpu", torch.float32, 5, 12, 1e-5)
    g = torch.Generator().manual_seed(0)
    x, w = torch.randn(4, 12, generator=g).double(), torch.randn(12, generator=g).double()
    z = torch.full_like(x, 200.0)                       # a gate of one
    for parts in (1, 2, 6):
        got = MX.part_norm_linear(x.float(), w.float(), parts, 1e-5, torch.eye(12))
        assert torch.allclose(got.double(), plain.part_norm(x / 200.0, z, w, parts, 1e-5), atol=1e-5)


def test_plain_gated_feed_forward():
    h = torch.randn(3, 10, dtype=torch.float32)
    assert torch.allclose(MX.clamped_glu(h, float("inf"), 1.0, 0.0), torch.nn.functional.silu(h[:, :5]) * h[:, 5:], atol=1e-6)


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


@pytest.mark.parametrize("kind", ["attention", "ssm"])
def test_models_of_one_kind_of_layer(kind):
    """No states, or no pages: the engine keeps what the layers need."""
    mixers = [attn(), attn(kv_from=0)] if kind == "attention" else [ssm(), ssm(heads=2, groups=1, norm_groups=2)]
    cfg = plain.make_config([layer(mixers[0], ff()), layer(mixers[1], moe())])
    e = cases.sizes_for_all(F32, cfg, 40, [[40], [25] + [1] * 15], 3e-5, seed=2)
    assert len(e.kv.layers) == (1 if kind == "attention" else 0) and (e.states is None) == (kind == "attention")
    assert (e.prefix_cache is not None) == (kind == "attention")


def test_a_layer_on_anothers_keys_keeps_none():
    e = U.engine_for(cases.config_a(), plain.make_weights(cases.config_a()), **F32)
    assert set(e.kv.layers) == {1} and set(e.states.layers) == {0, 2, 4, (0, "conv"), (2, "conv")}      # one tap looks at nothing back


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
    cfg = plain.make_config([layer(attn(), ff()), layer(attn(kv_from=0), moe())])
    W = plain.make_weights(cfg, 13)
    e = U.engine_for(cfg, W, **F32)
    prompt = U.tokens_for(cfg, 40, 6)
    for tail in ([], [3, 4, 5]):
        p = prompt + tail
        assert e.generate(p, {"temperature": 0.0, "max_new_tokens": 6})["output_ids"] == cases.greedy(cfg, W, p, 6)
    assert e.stats.get("prefix_cache_hit_tokens", 0) >= 32


def test_routed_experts_are_recorded():
    """One row per token and layer with experts, as wide as the widest layer."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 8)
    e = U.engine_for(cfg, W, **F32)
    r = e.add_request(U.tokens_for(cfg, 20, 2), {"temperature": 0.0, "max_new_tokens": 5}, return_routed_experts=True)
    while not r.done.is_set():
        e.step()
    import numpy as np

    got, xs = np.concatenate(r.routed)[:24], []
    plain.run(cfg, W, (r.input_ids + r.output_ids)[:24], layers=xs)
    for col, i in enumerate((1, 3, 4)):
        Wd, f = {k: v.double() for k, v in W.items()}, cfg["layers"][i]["mlp"]
        h = plain.rms(xs[i - 1], cfg["norm"]["eps"]) * (1 + Wd[f"l{i}.norm2"])
        idx, _ = plain.choose(h @ Wd[f"l{i}.mlp.router"].T, Wd[f"l{i}.mlp.correction"], f["router"])
        k = f["router"]["top"]
        assert np.array_equal(np.sort(got[:, col, :k]), np.sort(idx.numpy())) and (got[:, col, k:] == -1).all(), i
    assert got.shape[1] == 3


def test_scoring_a_prompt():
    """The logits' scale counts wherever rows meet the head."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 8)
    e = U.engine_for(cfg, W, **F32)
    toks = U.tokens_for(cfg, 25, 2)
    r = e.add_request(toks, {"temperature": 0.0, "max_new_tokens": 1}, logprob_start_len=0)
    while not r.done.is_set():
        e.step()
    lp = torch.log_softmax(plain.run(cfg, W, toks), -1)
    assert r.input_logprobs == pytest.approx([float(lp[i, toks[i + 1]]) for i in range(24)], abs=1e-4)


def test_memory_release_and_weight_update_keep_the_model():
    cfg = cases.config_a()
    W, W2 = plain.make_weights(cfg, 9), plain.make_weights(cfg, 10)
    e = U.engine_for(cfg, W, **F32)
    toks = U.tokens_for(cfg, 20, 3)
    e.release_memory_occupation()
    e.resume_memory_occupation()
    e.update_weights_from_tensor([kv for n, t in hf_state_to_ours(W2, e.cfg).items() for kv in to_hf(n, t, e.cfg)], weight_version=3)
    assert U.rel(U.feed_alone(e, toks, [12, 1, 7]), plain.run(cfg, W2, toks)) < 2e-5
