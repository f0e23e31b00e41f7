"""Ronupel on the CPU: configuration and names, the mechanisms' statements, cache / batching of the engine, loops, generation."""
from __future__ import annotations

import json
import os

import pytest
import torch

import layered_utils as U
import plain_ronupel as plain
import ronupel_cases as cases
from miles_b200.models import designs, ronupel
from miles_b200.models.config import ModelConfig, get_config
from miles_b200.models.convert import hf_state_to_ours, load_named_into_model, to_hf
from miles_b200.models.layered import AttentionSpec, LayeredModel, LinearScaling, LoopSpec, Rotary
from miles_b200.models.qwen3 import build_model
from miles_b200.ops import mixers as MX
from miles_b200.ops import mixers_reference as ref

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
        assert c.family == "ronupel" and c.block == "parallel" and c.tie_embeddings
        assert ronupel.from_config(c.to_hf_config()) == c
    c = ModelConfig.from_hf_config(cases.config_a())
    assert c.loop == LoopSpec(1, 3, 3) and c.layer_specs[2].mlp is None and c.layer_specs[1].mlp.shared is None
    assert c.runs() == plain.order_of_runs(cases.config_a()) and len(c.runs()) == 8
    assert c.num_experts == 7 and c.moe_topk == 3 and c.num_moe_layers == 5
    c.save(str(tmp_path))
    assert get_config(str(tmp_path)) == c
    assert isinstance(build_model(c, dtype=torch.float32), LayeredModel)
    assert get_config("ronupel-tiny").family == "ronupel" and "Ronupel" == designs.DESIGNS["ronupel"].ARCHITECTURE
    for change in ({"type": "other"}, {"mlp": {"kind": "other"}}):
        cfg = cases.config_a()
        cfg["layers"][0].update(change)
        with pytest.raises(ValueError):
            ronupel.from_config(cfg)
    cfg = cases.config_a()
    cfg["loop"]["stop"] = 9
    with pytest.raises(AssertionError):
        build_model(ronupel.from_config(cfg))


def test_fewer_layers_keep_a_valid_loop():
    c = ModelConfig.from_hf_config(cases.config_a())
    assert c.with_(num_layers=2).loop == LoopSpec(1, 2, 3) and c.with_(num_layers=1).loop is None
    assert [l for l, _ in c.with_(num_layers=2).runs()] == [0, 1, 1, 1]


def test_checkpoint_names_round_trip():
    cfg = cases.config_a()
    c, W = ronupel.from_config(cfg), plain.make_weights(cfg)
    ours = hf_state_to_ours(W, c)
    model = build_model(c, dtype=torch.bfloat16)
    assert set(ours) == {n for n, _ in model.named_parameters()}
    for n, p in model.named_parameters():
        assert tuple(p.shape) == tuple(ours[n].shape) == designs.param_shapes(c)[n], n
    back = dict(kv for n, t in ours.items() for kv in to_hf(n, t, c))
    assert set(back) == set(W) and all(torch.equal(back[n], W[n]) for n in W)
    assert c.num_params() == sum(t.numel() for t in W.values())
    # a token meets the looped layers three times and only its own experts
    seen = sum(t.numel() * (3 if n[:3] in ("l1.", "l2.") else 1) for n, t in W.items())
    seen -= 3 * 64 * ((5 - 2) * 56 + 3 * (3 - 3) * 24 + (7 - 1) * 40)
    assert c.num_params(active_only=True) == seen


def test_weights_in_any_portions():
    """A weight stream may cut stacked projections and experts anywhere between tensors."""
    cfg = cases.config_a()
    c, W = ronupel.from_config(cfg), plain.make_weights(cfg, 12)
    from miles_b200.parallel.state import ParallelState

    model = build_model(c, dtype=torch.float32)
    whole = hf_state_to_ours(W, c)
    for name, t in reversed(list(W.items())):
        load_named_into_model(model, [(name, t)], c, ParallelState.single())
    for n, p in model.named_parameters():
        assert torch.equal(p.data, whole[n].float()), n
    assert load_named_into_model(model, list(whole.items()), c, ParallelState.single()) == set(whole)
    with pytest.raises(AssertionError, match="configuration says"):
        load_named_into_model(model, [("l0.mlp.e1.up", torch.zeros(2, 2))], c, ParallelState.single())


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
    del W["l1.mlp.e2.up"]
    save_safetensors(str(tmp_path / "model.safetensors"), W)
    with pytest.raises(ValueError, match="lacks"):
        e.update_weights_from_disk(str(tmp_path))


def test_serving_build_of_a_configuration():
    from miles_b200.ops import build

    assert build.serve_kind(get_config("ronupel-tiny")) == "attention_experts_prep" and build.serve_kind(get_config("nopelorn-tiny")) == "latent_linear"
    for kind, files in build.SERVE_PARTS.items():
        assert all(os.path.exists(os.path.join(build.CSRC, f)) for f in build.SERVE_SOURCES + files), kind


# ---- mechanisms ---------------------------------------------------------------------------------------------------------------

def test_linear_scaling_of_the_rotation():
    f, mag = Rotary(500.0, 8, LinearScaling(2.5)).table()
    assert mag == 1.0 and f == pytest.approx([500.0 ** (-i / 4) / 2.5 for i in range(4)], rel=1e-14)
    x = torch.randn(7, 3, 8, dtype=torch.float64)
    pos = torch.tensor([0, 1, 5, 100, 3, 3, 1000])
    got = ref.rotate_pairs(x, pos, torch.tensor(f, dtype=torch.float64), 1.0)
    assert torch.allclose(got, plain.rotate(x, pos, {"base": 500.0, "dims": 8, "scaling": {"factor": 2.5}}), atol=1e-6)


def test_edges_and_sinks():
    m = plain.mixer_spec(scale=3.0 / 24 ** 0.5)
    cases.edges("cpu", torch.float32, m, 60, 1e-4, [[60], [59, 1], [7, 2, 20]])
    cases.sinks("cpu", torch.float32, m, 40, 1e-5)


@pytest.mark.parametrize("T,E,k,D,F", [(9, 5, 2, 16, 12), (1, 1, 1, 7, 5), (30, 3, 3, 8, 10)])
def test_experts(T, E, k, D, F):
    cases.experts("cpu", torch.float32, T, E, k, D, F, 1e-5)
    z = torch.randn(T, E, generator=torch.Generator().manual_seed(1))
    w, idx = ref.topk_softmax(z, k)
    pi, pw = plain.choose(z.double(), k)
    assert torch.equal(idx.long(), pi) and torch.allclose(w.double(), pw, atol=1e-6)


def test_sum_and_norm():
    g = torch.Generator().manual_seed(0)
    x, a, b, extra = (torch.randn(5, 12, generator=g) for _ in range(4))
    nw, to = torch.randn(12, generator=g), torch.empty(5, 12)
    h = MX.sum_norm(x, to, [MX.Addend(a), MX.Addend(b)], extra, nw, 1e-5)
    want = x.double() + a + b + extra
    assert torch.allclose(to.double(), want, atol=1e-6) and torch.allclose(h.double(), plain.rms(want, nw.double(), 1e-5), atol=1e-5)


# ---- the model in the engine -----------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name,T", [("a", 75), ("b", 61)])
def test_pieces_of_any_size(name, T):
    cfg = getattr(cases, f"config_{name}")()
    cases.sizes_for_all(F32, cfg, T, [[T], [T - 20] + [1] * 20, [2], [1, 30, 2, 3, 9, 17]], 3e-5)


def test_residual_after_every_layer_run():
    cfg = cases.config_a()
    W, toks, want = plain.make_weights(cfg, 7), U.tokens_for(cfg, 30, 1), []
    plain.run(cfg, W, toks, layers=want)
    e = U.engine_for(cfg, W, **F32)
    e.record_residual = got = []
    U.feed_alone(e, toks, [30])
    assert len(got) == len(want) == 8
    for a, b in zip(got, want):
        assert U.rel(a, b) < 1e-5


@pytest.mark.parametrize("loop", [None, (0, 4, 1), (0, 4, 2), (3, 4, 3), (0, 1, 2)])
def test_loops(loop):
    """Any range, any number of passes; every pass has a cache of its own (decoding reads all of them)."""
    cfg = dict(cases.config_a(), loop=dict(zip(("start", "stop", "times"), loop)) if loop else None)
    e = cases.sizes_for_all(F32, cfg, 40, [[40], [25] + [1] * 15], 3e-5, seed=2)
    assert len(e.kv.layers) == len(plain.order_of_runs(cfg))


def test_mixed_batches_reuse_pages():
    cases.mixed_batches(dict(F32, blocks=16), cases.config_a(), [70, 41, 5, 66, 1, 30], 3e-5)


def test_first_tokens_stay_in_sight():
    """Sequences that differ in their first token only differ at the end, far outside the windows: through the kept tokens."""
    cfg = plain.make_config([plain.layer_spec(window=5, keep=1, experts=0, scale=0.02)])
    W = plain.make_weights(cfg, 2)
    W["l0.mix.sink"].fill_(-20.0)
    e = U.engine_for(cfg, W, **F32)
    rest, ends = U.tokens_for(cfg, 40, 3), []
    for first in (0, 5):
        toks = [first] + rest
        want = plain.run(cfg, W, toks)
        for sizes in ([41], [1] * 41, [2, 39]):
            got = U.feed_alone(e, toks, sizes)
            assert U.rel(got, want) < 2e-5
        ends.append(want[-1])
    assert float((ends[0] - ends[1]).abs().max()) > 0.1


# ---- scheduler ------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("kw", [{}, {"chunked_prefill_size": 16}, {"chunked_prefill_size": 16, "mixed_batches": True},
                                {"share_prompt_kv": False, "mixed_batches": True, "prefix_cache": False}])
def test_greedy_generation(kw):
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 5)
    prompts = [U.tokens_for(cfg, n, n) for n in (37, 3, 20)]
    prompts.append(list(prompts[2]))                      # an identical prompt: shares pages
    want = [cases.greedy(cfg, W, p, 10) for p in prompts[:3]]
    e = U.engine_for(cfg, W, slots=3, **F32, **kw)          # fewer slots than requests: a later one waits and joins while others run
    lengths = [10, 6, 10, 10]
    out = e.generate(prompts, [{"temperature": 0.0, "max_new_tokens": n} for n in lengths])
    assert [o["output_ids"] for o in out] == [w[:n] for w, n in zip(want + [want[2]], lengths)]
    if kw.get("mixed_batches"):
        assert e.stats.get("mixed_steps", 0) > 0


def test_shared_prefixes_come_from_the_cache():
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 13)
    e = U.engine_for(cfg, W, **F32)
    prompt = U.tokens_for(cfg, 40, 6)
    for tail in ([], [3, 4, 5]):
        p = prompt + tail
        assert e.generate(p, {"temperature": 0.0, "max_new_tokens": 6})["output_ids"] == cases.greedy(cfg, W, p, 6)
    assert e.stats.get("prefix_cache_hit_tokens", 0) >= 32


def test_retraction():
    """Too few pages for all: a request loses its pages, starts again from its prompt and output, same tokens."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 6)
    prompts = [U.tokens_for(cfg, n, 40 + n) for n in (30, 29, 31)]
    want = [cases.greedy(cfg, W, p, 14) for p in prompts]
    e = U.engine_for(cfg, W, blocks=7, context=60, prefix_cache=False, **F32)
    out = e.generate(prompts, {"temperature": 0.0, "max_new_tokens": 14})
    assert [o["output_ids"] for o in out] == want and e.stats["retractions"] > 0


@pytest.mark.parametrize("kw", [{}, {"chunked_prefill_size": 7, "mixed_batches": True}])
def test_routed_experts_of_every_layer_run(kw):
    """What the engine records of the routing: one row per token and layer run with experts, as wide as the widest layer."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 8)
    e = U.engine_for(cfg, W, **F32, **kw)
    r = e.add_request(U.tokens_for(cfg, 20, 2), {"temperature": 0.0, "max_new_tokens": 5}, return_routed_experts=True)
    other = e.add_request(U.tokens_for(cfg, 11, 3), {"temperature": 0.0, "max_new_tokens": 9})
    while not (r.done.is_set() and other.done.is_set()):
        e.step()
    import numpy as np

    got = np.concatenate(r.routed)[:24]
    toks, Wd = (r.input_ids + r.output_ids)[:24], {k: v.double() for k, v in W.items()}
    x = first = Wd["embed"][torch.tensor(toks)]
    col = 0
    for i, again in plain.order_of_runs(cfg):
        x = x + first if again else x
        f, h = cfg["layers"][i]["mlp"], plain.rms(x, Wd[f"l{i}.norm1"], cfg["norm"]["eps"])
        y = plain.attention(h, Wd, f"l{i}.mix.", cfg["layers"][i]["mixer"], cfg["norm"]["eps"])
        if f is not None:
            idx, _ = plain.choose(h @ Wd[f"l{i}.mlp.router"].T + Wd[f"l{i}.mlp.router.b"], f["router"]["top"])
            k = f["router"]["top"]
            assert np.array_equal(got[:, col, :k], idx.numpy()) and (got[:, col, k:] == -1).all(), (i, col)
            y, col = y + plain.mixture(h, Wd, f"l{i}.mlp.", f), col + 1
        x = x + y
    assert col == got.shape[1] == e.model.num_moe_layers == 5


def test_scoring_a_prompt():
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 8)
    e = U.engine_for(cfg, W, **F32)
    toks = U.tokens_for(cfg, 25, 2)
    r = e.add_request(toks, {"temperature": 0.0, "max_new_tokens": 1}, logprob_start_len=0)
    while not r.done.is_set():
        e.step()
    lp = torch.log_softmax(plain.run(cfg, W, toks), -1)
    assert r.input_logprobs == pytest.approx([float(lp[i, toks[i + 1]]) for i in range(24)], abs=1e-4)
    with pytest.raises(NotImplementedError):
        e.add_prefilled(toks, 1, 0.0, torch.zeros(1))


def test_memory_release_and_weight_update_keep_the_model():
    cfg = cases.config_a()
    W, W2 = plain.make_weights(cfg, 9), plain.make_weights(cfg, 10)
    e = U.engine_for(cfg, W, **F32)
    toks = U.tokens_for(cfg, 20, 3)
    e.release_memory_occupation()
    e.resume_memory_occupation()
    e.update_weights_from_tensor([kv for n, t in hf_state_to_ours(W2, e.cfg).items() for kv in to_hf(n, t, e.cfg)], weight_version=3)
    assert U.rel(U.feed_alone(e, toks, [12, 1, 7]), plain.run(cfg, W2, toks)) < 2e-5


def test_attention_mixer_in_the_other_arrangement():
    """The mixer is not tied to the parallel block: beside linear attention, with norms on the outputs and a dense feed-forward."""
    from miles_b200.engine.engine import Engine
    from miles_b200.models.layered import GluSpec, LayeredConfig, LayerSpec, LinearStateSpec

    c = LayeredConfig(name="mixed", family="nopelorn", vocab_size=50, hidden_size=32, num_layers=2, num_heads=1, num_kv_heads=1, head_dim=0,
                      ffn_hidden_size=0, layer_specs=(LayerSpec(AttentionSpec(4, 2, 8, 8, 0.3, Rotary(100.0, 4), 9, 2), GluSpec(24, 2.0)),
                                                      LayerSpec(LinearStateSpec(2, 8, 8, (0.9, 0.8)), None)))
    e = Engine(c, num_blocks=8, block_size=16, max_running_requests=2, max_context_len=64, **F32)
    toks = U.tokens_for({"vocab": 50}, 30)
    whole = U.feed_alone(e, toks, [30])
    for sizes in ([1] * 30, [9, 2, 19]):
        assert U.rel(U.feed_alone(e, toks, sizes), whole) < 1e-5
