"""Nopelorn on the CPU: configuration and names, the mechanisms' statements, cache / state / batching of the engine, generation."""
from __future__ import annotations

import json
import os

import pytest
import torch

import layered_utils as U
import nopelorn_cases as cases
import plain_nopelorn as plain
from miles_b200.models import nopelorn
from miles_b200.models.config import ModelConfig, get_config
from miles_b200.models.convert import hf_state_to_ours, to_hf
from miles_b200.models.layered import LayeredModel, LatentSpec
from miles_b200.models.qwen3 import build_model

F32 = dict(device="cpu", dtype=torch.float32)


@pytest.fixture(autouse=True)
def _few_threads():
    n = torch.get_num_threads()
    torch.set_num_threads(min(n, 4))
    yield
    torch.set_num_threads(n)


# ---- configuration, names, files ----------------------------------------------------------------------------------------

def test_config_round_trip_and_registry(tmp_path):
    cfg = cases.config_a()
    c = ModelConfig.from_hf_config(cfg)
    assert c.family == "nopelorn" and c.num_layers == 4 and c.layer_specs[2].mixer.kv_from == 1 and c.layer_specs[3].mlp is None
    again = nopelorn.from_config(c.to_hf_config())
    assert again == c
    c.save(str(tmp_path))
    assert get_config(str(tmp_path)) == c
    assert isinstance(build_model(c, dtype=torch.float32), LayeredModel)
    assert get_config("nopelorn-tiny").family == "nopelorn"
    with pytest.raises(ValueError):
        nopelorn.from_config({**cfg, "layers": [{**cfg["layers"][0], "type": "other"}]})


def test_checkpoint_names_round_trip():
    cfg = cases.config_a()
    c, W = nopelorn.from_config(cfg), plain.make_weights(cfg)
    ours = hf_state_to_ours(W, c)
    model = build_model(c, dtype=torch.bfloat16)
    assert set(ours) == {n for n, _ in model.named_parameters()}
    for n, p in model.named_parameters():
        assert tuple(p.shape) == tuple(ours[n].shape), n
    back = dict(kv for n, t in ours.items() for kv in to_hf(n, t, c))
    assert set(back) == set(W) and all(torch.equal(back[n], W[n]) for n in W)
    assert c.num_params() == sum(t.numel() for t in W.values())


def test_weights_in_any_portions():
    """A weight stream may cut a stacked projection anywhere between tensors."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 12)
    c = nopelorn.from_config(cfg)
    from miles_b200.models.convert import load_named_into_model
    from miles_b200.parallel.state import ParallelState

    model = build_model(c, dtype=torch.float32)
    whole = hf_state_to_ours(W, c)
    for name, t in reversed(list(W.items())):
        load_named_into_model(model, [(name, t)], c, ParallelState.single())
    for n, p in model.named_parameters():
        assert torch.equal(p.data, whole[n].float()), n
    assert load_named_into_model(model, list(whole.items()), c, ParallelState.single()) == set(whole)


def test_weights_from_disk(tmp_path):
    from miles_b200.checkpoint.hf_io import save_safetensors

    cfg = cases.config_b()
    W = plain.make_weights(cfg, 4)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_safetensors(str(tmp_path / "model.safetensors"), W)
    from miles_b200.engine.engine import Engine

    e = Engine(get_config(str(tmp_path)), num_blocks=8, max_running_requests=2, max_context_len=64, **F32)
    e.update_weights_from_disk(str(tmp_path))
    toks = U.tokens_for(cfg, 20)
    assert U.rel(U.feed_alone(e, toks, [20]), plain.run(cfg, W, toks)) < 1e-5
    del W["l1.mlp.up"]
    save_safetensors(str(tmp_path / "model.safetensors"), W)
    with pytest.raises(ValueError, match="lacks"):
        e.update_weights_from_disk(str(tmp_path))


def test_yarn_frequencies():
    for rot in (dict(base=10000.0, dims=32, scaling=dict(factor=8.0, original=4096, fast=32.0, slow=1.0)),
                dict(base=300.0, dims=6, scaling=dict(factor=1.0, original=16, fast=4.0, slow=4.0)),
                dict(base=5e5, dims=64, scaling=dict(factor=40.0, original=128, fast=64.0, slow=0.5)), dict(base=77.0, dims=10)):
        m = dict(plain.latent_spec()["mixer"], rot=rot, rot_dim=rot["dims"])
        f, mag = nopelorn._mixer("latent_attention", m).rotary.table()
        want, wm = plain.yarn_frequencies(rot)
        assert mag == pytest.approx(wm, rel=1e-14) and f == pytest.approx(want, rel=1e-14)


# ---- the model in the engine -----------------------------------------------------------------------------------------------

@pytest.mark.parametrize("name,T", [("a", 83), ("b", 61)])
def test_pieces_of_any_size(name, T):
    cfg = getattr(cases, f"config_{name}")()
    cases.sizes_for_all(F32, cfg, T, [[T], [T - 20] + [1] * 20, [2], [1, 30, 2, 3, 9, 17]], 2e-5)


def test_residual_after_every_layer():
    cfg = cases.config_a()
    W, toks, want = plain.make_weights(cfg, 7), U.tokens_for(cfg, 30, 1), []
    plain.run(cfg, W, toks, layers=want)
    e = U.engine_for(cfg, W, **F32)
    e.record_residual = got = []
    U.feed_alone(e, toks, [30])
    assert len(got) == 4
    for a, b in zip(got, want):
        assert U.rel(a, b) < 1e-5


def test_mixed_batches_reuse_pages_and_slots():
    cases.mixed_batches(dict(F32, blocks=16), cases.config_a(), [70, 41, 5, 66, 1, 30], 2e-5)


def test_window_edges_and_sink():
    m = plain.latent_spec(window=19)["mixer"]
    cases.window_edges("cpu", torch.float32, m, 60, 1e-4, [[60], [59, 1], [7, 2, 20]])
    cases.sink_counts("cpu", torch.float32, m, 40, 1e-5)


def test_linear_state_statement():
    cases.linear_state("cpu", torch.float32, 2, 8, 12, [50, 33, 7], [[(0, 20), (1, 9)], [(0, 1), (2, 1), (1, 1)], [(0, 2), (2, 4)],
                                                                    [(0, 40), (1, 40), (2, 40)]], 1e-5, pull=(0, 49))


def test_first_tokens_and_bigram():
    """Two sequences that differ in their first token only: everything after depends on it (state, bigram of the second token); a
    sequence's first token takes the table's last row whatever was fed before it."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 2)
    e = U.engine_for(cfg, W, **F32)
    for first in (0, 5):
        toks = [first] + U.tokens_for(cfg, 12, 3)
        for sizes in ([13], [1] * 13, [2, 11]):
            assert U.rel(U.feed_alone(e, toks, sizes), plain.run(cfg, W, toks)) < 2e-5
    # a very large bigram product stays exact
    big = dict(cfg, embedding={"bigram": {"buckets": 91, "mul_prev": 2 ** 31 - 1, "mul_cur": 10 ** 9 + 7}})
    W = plain.make_weights(big, 2)
    toks = U.tokens_for(big, 20, 5)
    assert U.rel(U.feed_alone(U.engine_for(big, W, **F32), toks, [20]), plain.run(big, W, toks)) < 2e-5


# ---- scheduler ------------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("kw", [{}, {"chunked_prefill_size": 16}, {"chunked_prefill_size": 16, "mixed_batches": True},
                                {"share_prompt_kv": False, "mixed_batches": True}])
def test_greedy_generation(kw):
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 5)
    prompts = [U.tokens_for(cfg, n, n) for n in (37, 3, 20)]
    prompts.append(list(prompts[2]))                      # an identical prompt: shares pages and copies the state
    want = [cases.greedy(cfg, W, p, 12)[0] for p in prompts[:3]]
    e = U.engine_for(cfg, W, slots=3, **F32, **kw)          # fewer slots than requests: a later one waits for a slot
    lengths = [12, 7, 12, 12]                               # … and joins while others run
    out = e.generate(prompts, [{"temperature": 0.0, "max_new_tokens": n} for n in lengths])
    assert [o["output_ids"] for o in out] == [w[:n] for w, n in zip(want + [want[2]], lengths)]
    assert e.allocator.num_free == 24 and e.states.num_free == 3
    if kw.get("mixed_batches"):
        assert e.stats.get("mixed_steps", 0) > 0


def test_models_with_one_kind_of_layer():
    """Only latent attention: no state slots, and shared prefixes come from the cache.  Only linear attention: no cached rows."""
    cfg = plain.make_config([plain.latent_spec(window=19), plain.latent_spec(heads=2, window=50, kv_from=0)])
    W = plain.make_weights(cfg, 13)
    e = U.engine_for(cfg, W, **F32)
    assert e.states is None and e.prefix_cache is not None
    prompt = U.tokens_for(cfg, 40, 6)
    for tail in ([], [3, 4, 5]):
        p = prompt + tail
        out = e.generate(p, {"temperature": 0.0, "max_new_tokens": 8})
        assert out["output_ids"] == cases.greedy(cfg, W, p, 8)[0]
    assert e.stats.get("prefix_cache_hit_tokens", 0) >= 32
    cfg = plain.make_config([plain.lightning_spec(), plain.lightning_spec(heads=3, dim=4, vdim=20, ff=None)])
    W = plain.make_weights(cfg, 14)
    e = U.engine_for(cfg, W, **F32)
    assert not e.kv.layers and e.kv.allocated and e.prefix_cache is None
    p = U.tokens_for(cfg, 30, 7)
    assert e.generate(p, {"temperature": 0.0, "max_new_tokens": 8})["output_ids"] == cases.greedy(cfg, W, p, 8)[0]


def test_retraction_restarts_the_state():
    """Too few pages for all: a request loses its pages and slot, starts again from its prompt and output, same tokens."""
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 6)
    prompts = [U.tokens_for(cfg, n, 40 + n) for n in (30, 29, 31)]
    want = [cases.greedy(cfg, W, p, 20)[0] for p in prompts]
    e = U.engine_for(cfg, W, blocks=9, context=60, **F32)
    out = e.generate(prompts, {"temperature": 0.0, "max_new_tokens": 20})
    assert [o["output_ids"] for o in out] == want
    assert e.stats["retractions"] > 0 and e.states.num_free == 4


def test_scoring_a_prompt_and_limits():
    cfg = cases.config_a()
    W = plain.make_weights(cfg, 8)
    e = U.engine_for(cfg, W, **F32)
    toks = U.tokens_for(cfg, 25, 2)
    r = e.add_request(toks, {"temperature": 0.0, "max_new_tokens": 1}, logprob_start_len=0)
    while not r.done.is_set():
        e.step()
    lp = torch.log_softmax(plain.run(cfg, W, toks), -1)
    assert r.input_logprobs == pytest.approx([float(lp[i, toks[i + 1]]) for i in range(24)], abs=1e-4)
    a = e.open_request("a")
    with pytest.raises(ValueError):
        e.open_request("a")
    with pytest.raises(ValueError):
        e.feed([(a, [cfg["vocab"]], [])])
    with pytest.raises(ValueError):
        e.feed([(a, [1, 2], [2])])
    for n in "bcd":
        e.open_request(n)
    with pytest.raises(RuntimeError):
        e.open_request("e")
    for n in "abcd":
        e.close_request(n)
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
    assert e.get_weight_version() == 3


def test_replay_writes_logits(tmp_path):
    from miles_b200.engine.trace import replay

    cfg = cases.config_a()
    W = plain.make_weights(cfg, 11)
    e = U.engine_for(cfg, W, **F32)
    x, y = U.tokens_for(cfg, 20, 1), U.tokens_for(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": x[:13], "want": [0, 12]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": y, "want": [8]}, {"id": "p", "tokens": x[13:14], "want": [0]}], "end": ["q"]},
             {"step": 2, "entries": [{"id": "p", "tokens": x[14:15], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "p", "tokens": x[15:], "want": [4]}], "end": ["p"]}]
    said = []
    replay(e, [json.dumps(s) + "\n" for s in steps], str(tmp_path), said.append)
    assert said == [f"done {i}" for i in range(4)] and sorted(os.listdir(tmp_path)) == ["0.f32", "1.f32", "3.f32"]
    wx, wy = plain.run(cfg, W, x), plain.run(cfg, W, y)

    def rows(i):
        return torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])

    assert U.rel(rows(0), wx[[0, 12]]) < 2e-5 and U.rel(rows(1), torch.stack([wy[8], wx[13]])) < 2e-5 and U.rel(rows(3), wx[[19]]) < 2e-5
    assert e.states.num_free == 4 and isinstance(e.cfg.layer_specs[1].mixer, LatentSpec)
