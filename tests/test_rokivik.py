"""Rokivik models on the framework's CPU configuration (PyTorch path, the engine's real scheduler and cache manager) against
a plain restatement of the equations."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import oracle_rokivik as O  # noqa: E402
from rokivik_cases import CASES, config, feed_all, latent, load, mamba, rel, sharpen, tokens_of, with_window  # noqa: E402

from miles_b200.engine import SamplingParams  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 2e-5


@pytest.fixture(scope="module", params=list(CASES))
def case(request, tmp_path_factory):
    cfg = CASES[request.param]
    W = O.random_weights(cfg, seed=3, dtype=torch.float32)
    return cfg, W, load(cfg, W, tmp_path_factory.mktemp("m"), "cpu", torch.float32)


def test_whole_prompt_single_tokens_and_portions(case):
    cfg, W, eng = case
    toks = tokens_of(61, cfg["vocab"], 1)
    want = O.model(cfg, W, toks)
    for cuts in ([61], [1], [2], [3, 2, 7, 2, 11], [8], [40, 1]):
        assert rel(feed_all(eng, "a", toks, cuts), want) < TOL, cuts


def test_unequal_batch_equals_each_alone(case):
    cfg, W, eng = case
    seqs = {f"s{n}": tokens_of(n, cfg["vocab"], n) for n in (3, 1, 37, 16)}
    got = eng.feed([(k, t[:max(1, len(t) - 3)], [max(1, len(t) - 3) - 1]) for k, t in seqs.items()])
    for (k, t), g in zip(seqs.items(), got):
        assert rel(g.cpu(), O.model(cfg, W, t)[max(1, len(t) - 3) - 1:max(1, len(t) - 3)]) < TOL
    # a decode step and a portion in the same call, rows in another order
    rest = [(k, seqs[k][len(seqs[k]) - 3:][:n], list(range(n))) for k, n in (("s37", 1), ("s16", 3))]
    for (k, t, _), g in zip(rest, eng.feed(rest)):
        n = len(seqs[k]) - 3
        assert rel(g.cpu(), O.model(cfg, W, seqs[k][:n + len(t)])[n:]) < TOL
    for k in seqs:
        eng.end_feed(k)


def test_pages_and_state_rows_are_used_again(case):
    cfg, W, eng = case
    free, rows = eng.pool.num_free, len(eng.slots_free)
    for r in range(6):
        toks = tokens_of(20 + 9 * r, cfg["vocab"], 50 + r)
        assert rel(feed_all(eng, f"r{r}", toks, [13, 1, 5]), O.model(cfg, W, toks)) < TOL
    assert (eng.pool.num_free, len(eng.slots_free)) == (free, rows)


def test_greedy_generation_through_the_scheduler(case):
    """More requests than rows, a page pool that runs dry (retraction), prompts in portions of 7 tokens."""
    cfg, W, eng0 = case
    import miles_b200.engine as E

    eng = E.Engine(eng0.model, max_running=3, num_pages=22, page_size=8, max_seq_len=96, max_prefill_tokens=7)
    prompts = [tokens_of(n, cfg["vocab"], n) for n in (30, 5, 44, 17, 23)]
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=40))
    assert eng.pool.num_free == 21 and len(eng.slots_free) == 3
    for p, o in zip(prompts, outs):
        ids = o["output_ids"]
        assert len(ids) == 40
        lg = O.model(cfg, W, p + ids[:-1])[len(p) - 1:]
        best = lg.max(-1).values
        got = lg.gather(1, torch.tensor(ids)[:, None])[:, 0]
        assert (best - got).max() < 1e-3 * lg.std()
        lp = torch.tensor([v for v, _ in o["meta_info"]["output_token_logprobs"]])
        assert torch.isfinite(lp).all()


def test_scoring_matches_generation_inputs(case):
    cfg, W, eng = case
    toks = tokens_of(25, cfg["vocab"], 9)
    want = torch.log_softmax(O.model(cfg, W, toks), -1)[:-1].gather(1, torch.tensor(toks[1:])[:, None])[:, 0]
    got = torch.tensor(eng.score(toks)["logprobs"][1:])
    assert (got - want).abs().max() < 1e-3


def test_abort_and_pause_in_the_middle_of_a_prompt(tmp_path):
    cfg = CASES["mixed"]
    W = O.random_weights(cfg, seed=5, dtype=torch.float32)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32, max_prefill_tokens=6)
    toks = tokens_of(40, cfg["vocab"], 2)
    eng.add_request(toks, SamplingParams(temperature=0.0, max_new_tokens=4), rid="x")
    eng.step()
    assert [r.rid for r in eng.prefilling] == ["x"] and not eng.running
    eng.pause_generation("retract")
    assert not eng.prefilling and eng.pool.num_free == 63
    eng.continue_generation()
    eng.step()
    assert eng.abort_request("x") == 1 and not eng.has_work() and eng.pool.num_free == 63
    eng.pop_finished()
    out = eng.generate([toks], SamplingParams(temperature=0.0, max_new_tokens=4))[0]["output_ids"]
    lg = O.model(cfg, W, toks + out[:-1])[-4:]
    assert (lg.max(-1).values - lg.gather(1, torch.tensor(out)[:, None])[:, 0]).max() < 1e-3


# ------------------------------------------------------------------------------------------------ edges that random weights hide
@pytest.mark.parametrize("window", [1, 2, 7, 8, 9, 16, 31])
def test_window_edges_in_prompts_and_decoding(tmp_path, window):
    """Sharp attention over one layer: the oracle with a window one longer or one shorter is far away."""
    cfg = config([latent(window=window, heads=4)])
    W = sharpen(cfg, O.random_weights(cfg, seed=window, dtype=torch.float32), 6.0)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    toks = tokens_of(50, cfg["vocab"], 4)
    want = O.model(cfg, W, toks)
    for cuts in ([50], [window], [20, 1], [window + 1, 2]):
        got = feed_all(eng, "a", toks, cuts)
        assert rel(got, want) < 10 * TOL
        assert rel(got, O.model(with_window(cfg, 1), W, toks)) > 0.05
        if window > 1:
            assert rel(got, O.model(with_window(cfg, -1), W, toks)) > 0.05


@pytest.mark.parametrize("back", [0, 1, 8, 23, 24, 25])
def test_one_far_token_is_seen_just_inside_the_window_only(tmp_path, back):
    cfg = config([latent(window=24)])
    W = O.random_weights(cfg, seed=1, dtype=torch.float32)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    toks = tokens_of(60, cfg["vocab"], 6)
    other = list(toks)
    other[55 - back] = (toks[55 - back] + 1) % cfg["vocab"]
    for cuts in ([60], [55, 1]):
        d = (feed_all(eng, "a", toks, cuts)[55] - feed_all(eng, "b", other, cuts)[55]).abs().max()
        assert (d > 1e-2) if back < 24 else (d < 1e-5)


def test_first_tokens_and_state_carry_over(tmp_path):
    """A slow state (decay near 1) still carries the first token far away; losing it at a portion's edge shows."""
    cfg = config([mamba(heads=2, groups=1, norm_groups=1)])
    W = O.random_weights(cfg, seed=8, dtype=torch.float32)
    W["l0.mix.A_log"] = torch.full((2,), -6.0)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    toks = tokens_of(80, cfg["vocab"], 3)
    want = O.model(cfg, W, toks)
    lost = O.model(cfg, W, toks[40:])
    for cuts in ([80], [40], [2], [1]):
        got = feed_all(eng, "a", toks, cuts)
        assert rel(got, want) < 5 * TOL and rel(got[40:], lost) > 0.05


def test_shared_latents_come_from_the_named_layer(tmp_path):
    cfg = CASES["attention"]
    W = O.random_weights(cfg, seed=2, dtype=torch.float32)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    assert eng.kv_cache[1][0].data_ptr() == eng.kv_cache[0][0].data_ptr()
    toks = tokens_of(30, cfg["vocab"], 1)
    W2 = dict(W)
    W2["l0.mix.dkv"] = W["l0.mix.dkv"].flip(0)
    assert rel(feed_all(eng, "a", toks, [30]), O.model(cfg, W2, toks)) > 0.05


def test_prefix_cache_and_handover_without_state(tmp_path):
    """Latents only: cached pages are shared between requests and travel to another engine; with state the cache is off."""
    cfg = CASES["attention"]
    W = O.random_weights(cfg, seed=2, dtype=torch.float32)
    a = load(cfg, W, tmp_path / "a", "cpu", torch.float32, prefix_cache=True, max_prefill_tokens=10)
    b = load(cfg, W, tmp_path / "b", "cpu", torch.float32, prefix_cache=True)
    plain = load(cfg, W, tmp_path / "c", "cpu", torch.float32)
    toks = tokens_of(45, cfg["vocab"], 1)
    sp = SamplingParams(temperature=0.0, max_new_tokens=12)
    want = plain.generate([toks], sp)[0]["output_ids"]
    assert a.generate([toks], sp)[0]["output_ids"] == want
    again = a.generate([toks], sp)[0]
    assert again["output_ids"] == want and again["meta_info"]["cached_tokens"] == 40
    assert b.import_prefix(a.export_prefix(toks)) >= 40
    got = b.generate([toks], sp)[0]
    assert got["output_ids"] == want and got["meta_info"]["cached_tokens"] == 40
    cfg = CASES["mixed"]
    assert load(cfg, O.random_weights(cfg, dtype=torch.float32), tmp_path / "d", "cpu", torch.float32, prefix_cache=True).prefix is None


# ------------------------------------------------------------------------------------------------ configuration, weights, command line
def test_configuration_round_trip_and_refusals(tmp_path):
    from miles_b200.models import ModelConfig

    for cfg in CASES.values():
        mc = ModelConfig.from_hf_config(cfg)
        assert mc.to_hf_config() == cfg and mc.family == "rokivik"
        n = 0
        for shape in O.tensor_shapes(cfg).values():
            k = 1
            for s in shape:
                k *= s
            n += k
        assert 0 <= mc.num_params() - n < 64 * (sum(1 for _ in cfg["layers"]) * 4) * cfg["width"]  # padding rows of fused weights only
    bad = config([latent(), latent(kv_from=0, kv_rank=40)])
    with pytest.raises(ValueError):
        ModelConfig.from_hf_config(bad)
    with pytest.raises(NotImplementedError):
        ModelConfig.from_hf_config(config([dict(latent(), type="other")]))


def test_weights_leave_under_checkpoint_names(tmp_path):
    from miles_b200.models.hf_mapping import hf_names, param_or_hf_view

    cfg = CASES["mixed"]
    W = O.random_weights(cfg, seed=3, dtype=torch.float32)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    out = dict(hf_names(eng.cfg, eng.store))
    assert set(out) == set(W) and all(torch.equal(out[k], W[k]) for k in W)
    param_or_hf_view(eng.cfg, eng.store, "l1.mlp.down").zero_()  # a weight update under a checkpoint name
    assert dict(hf_names(eng.cfg, eng.store))["l1.mlp.down"].abs().sum() == 0


def test_any_cache_dtype_and_layout_description():
    from miles_b200.models import ModelConfig
    from miles_b200.models.cache_layout import cache_layout

    lay = cache_layout(ModelConfig.from_hf_config(CASES["mixed"]), torch.bfloat16)
    assert lay.has_state and lay.layers[3].shares == 1
    assert lay.bytes_per_slot() == 2 * (40 + 64)
    assert lay.bytes_per_sequence() == 2 * (2 * 4 * (64 + 2 * 2 * 16) + 4 * 4 * 16 * 16)
    qwen = cache_layout(ModelConfig(), torch.float32)
    assert not qwen.has_state and qwen.bytes_per_slot() == 2 * 2 * 2 * 64 * 4


def test_trace_run_command(tmp_path):
    cfg = CASES["mixed"]
    W = O.random_weights(cfg, seed=11, dtype=torch.float32)
    d = O.write_checkpoint(tmp_path / "m", cfg, W)
    out = tmp_path / "out"
    out.mkdir()
    toks = tokens_of(12, cfg["vocab"], 1)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:7], "want": [2, 6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[7:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[8:], "want": [3]}], "end": ["a"]}]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(d), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "12", "--device", "cpu"], input="\n".join(json.dumps(s) for s in steps) + "\n", text=True, capture_output=True)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = O.model(cfg, W, toks)
    got = torch.frombuffer(bytearray((out / "0.f32").read_bytes() + (out / "2.f32").read_bytes()), dtype=torch.float32).view(3, -1)
    assert rel(got, want[[2, 6, 11]]) < TOL and not (out / "1.f32").exists()


def test_server_command_line_serves_the_design_and_training_refuses_it(tmp_path):
    from fastapi.testclient import TestClient

    from miles_b200.engine.server import build_app, build_from_args
    from miles_b200.utils.arguments import parse_args

    cfg = CASES["mixed"]
    W = O.random_weights(cfg, seed=3, dtype=torch.float32)
    d = O.write_checkpoint(tmp_path, cfg, W)
    engine, tokenizer, _ = build_from_args(["--hf-checkpoint", str(d), "--device", "cpu", "--max-running-requests", "2", "--page-size", "8",
                                            "--context-length", "64", "--max-prefill-tokens", "9"])
    assert tokenizer is None and engine.max_prefill_tokens == 9
    toks = tokens_of(21, cfg["vocab"], 1)
    with TestClient(build_app(engine)) as client:
        r = client.post("/generate", json={"input_ids": toks, "sampling_params": {"temperature": 0.0, "max_new_tokens": 5}}).json()
    lg = O.model(cfg, W, toks + r["output_ids"][:-1])[-5:]
    assert (lg.max(-1).values - lg.gather(1, torch.tensor(r["output_ids"])[:, None])[:, 0]).max() < 1e-3
    with pytest.raises(SystemExit):
        build_from_args(["--hf-checkpoint", str(d), "--device", "cpu", "--quantization", "mxfp8"])
    from miles_b200.utils.arguments import model_config_from_args

    with pytest.raises(NotImplementedError):
        model_config_from_args(parse_args(["--model-preset", "rokivik-smoke", "--num-rollout", "1", "--rollout-batch-size", "1"]))
