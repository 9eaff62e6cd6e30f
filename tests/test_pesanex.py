"""Pesanex models on the framework's CPU configuration (PyTorch path, the engine's real scheduler and cache manager) against a
plain restatement of the equations."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import oracle_pesanex as O  # noqa: E402
from oracle_rokivik import write_checkpoint  # noqa: E402
from pesanex_cases import CASES, RANKS, config, gla, parallel, retention, sharpen, slow  # noqa: E402
from rokivik_cases import feed_all, load, rel, row_errors, tokens_of  # noqa: E402

from miles_b200.engine import SamplingParams  # noqa: E402

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 3e-5


@pytest.fixture(scope="module", params=list(CASES))
def case(request, tmp_path_factory):
    cfg = CASES[request.param]
    W = O.random_weights(cfg, seed=3, dtype=torch.float32, rank=RANKS.get(request.param))
    return cfg, W, load(cfg, W, tmp_path_factory.mktemp("m"), "cpu", torch.float32)


def greedy_gap(cfg, W, prompt, ids):
    """How far below the best logit the generated tokens lie, over the spread of the logits."""
    lg = O.model(cfg, W, prompt + ids[:-1])[len(prompt) - 1:]
    return float((lg.max(-1).values - lg.gather(1, torch.tensor(ids)[:, None])[:, 0]).max() / lg.std())


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
        assert len(o["output_ids"]) == 40 and greedy_gap(cfg, W, p, o["output_ids"]) < 1e-3
        assert torch.isfinite(torch.tensor([v for v, _ in o["meta_info"]["output_token_logprobs"]])).all()


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
    assert greedy_gap(cfg, W, toks, out) < 1e-3


# ------------------------------------------------------------------------------------------------ what random weights would hide
def changed(cfg, **kw):
    """The configuration with a mixer's (or, in side-by-side layers, a side's) values replaced where it has them."""
    c = copy.deepcopy(cfg)
    for l in c["layers"]:
        for m in (l["mixer"], l["mixer"].get("left", {}), l["mixer"].get("right", {})):
            for k, v in kw.items():
                if k in m:
                    m[k] = v(m[k])
    return c


def shows(eng, cfg, W, wrong, toks, cuts=([50], [7], [20, 1])):
    """The engine follows the oracle and not a mistaken form of it."""
    want, off = O.model(cfg, W, toks), O.model(*wrong, toks)
    for c in cuts:
        got = feed_all(eng, "a", toks, c)
        assert rel(got, want) < 10 * TOL and rel(got, off) > 0.03, c


def test_constants_come_from_the_configuration(tmp_path):
    toks = tokens_of(50, 96, 4)
    half = lambda r: dict(r, dims=r["dims"] // 2)
    bases = lambda r: dict(r, base=r["base"] * 3)
    for k, (layer, kw) in enumerate([(parallel(), dict(scale=lambda s: 1.5 * s)), (parallel(), dict(rot=half)), (parallel(), dict(rot=bases)),
                                     (parallel(), dict(tau=lambda t: 2 * t)), (gla(), dict(tau=lambda t: t / 2)), (retention(), dict(rot=half)),
                                     (retention(), dict(rot=bases)), (retention(), dict(decay=lambda d: d[::-1]))]):
        cfg = config([layer])
        cfg, W = sharpen(cfg, O.random_weights(cfg, seed=k, dtype=torch.float32), 3.0)
        eng = load(cfg, W, tmp_path / str(k), "cpu", torch.float32)
        shows(eng, cfg, W, (changed(cfg, **kw), W), toks)


@pytest.mark.parametrize("sink", [-30.0, 0.0, 4.0])
def test_sink_counts_once_and_is_not_scaled(tmp_path, sink):
    cfg = config([parallel(scale=2.0, ff=0)])
    W = O.random_weights(cfg, seed=2, dtype=torch.float32)
    W["l0.mix.left.sink"] = torch.full((4,), sink)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    off = dict(W, **{"l0.mix.left.sink": torch.tensor([sink + 2.0, sink - 2.0, sink + 1.0, sink])})
    toks = tokens_of(50, cfg["vocab"], 4)
    want = O.model(cfg, W, toks)
    for c in ([50], [7], [20, 1]):
        got = feed_all(eng, "a", toks, c)
        assert rel(got, want) < 10 * TOL
        assert (rel(got, O.model(cfg, off, toks)) > 0.02) == (sink > -10)


def far_key(cfg, W, n, back):
    """Tokens whose last one attends, in one head of the first layer's left side, to a single token ``back`` places before it; and
    the same with that token replaced."""
    m, p, eps = cfg["layers"][0]["mixer"]["left"], "l0.mix.left.", cfg["norm"]["eps"]
    h = O.layer_norm(W["embed"], W["l0.norm1"], eps)
    q = O.unit_rms((h @ W[p + "q"].T).view(cfg["vocab"], m["heads"], -1)[:, 0, m["rot"]["dims"]:], eps)
    k = O.unit_rms((h @ W[p + "k"].T).view(cfg["vocab"], m["kv_heads"], -1)[:, 0, m["rot"]["dims"]:], eps)
    top = (q @ k.T).topk(2, -1)
    asks = int((top.values[:, 0] - top.values[:, 1]).argmax())
    key = int(top.indices[asks, 0])
    toks = [t if t != key else (key + 1) % cfg["vocab"] for t in tokens_of(n, cfg["vocab"], 6)]
    toks[n - 1] = asks
    other = list(toks)
    toks[n - 1 - back] = key
    return toks, other


@pytest.mark.parametrize("back", [1, 7, 8, 9, 30, 59])
def test_one_far_key_decides_a_row(tmp_path, back):
    """One key, anywhere before the last token, takes a head's weight: before and after page and portion borders, at the start."""
    cfg = config([parallel(scale=12.0, dims=2, ff=0)])
    W = O.random_weights(cfg, seed=1, dtype=torch.float32)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    toks, other = far_key(cfg, W, 60, back)
    a, b = O.model(cfg, W, toks), O.model(cfg, W, other)
    for cuts in ([60], [59, 1], [60 - back, 2], [4]):
        got = feed_all(eng, "a", toks, cuts)
        assert rel(got, a) < 30 * TOL and rel(got[59:], b[59:]) > 0.1, cuts


@pytest.mark.parametrize("layer", [retention(heads=2, decay=[1.0, 0.9999], ff=0), gla(), parallel(ff=0)], ids=["retention", "gla", "parallel"])
def test_first_tokens_and_state_carry_over(tmp_path, layer):
    """A slow state still carries the first token far away; losing it at a portion's edge shows."""
    cfg = config([layer])
    W = slow(O.random_weights(cfg, seed=8, dtype=torch.float32))
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    toks = tokens_of(80, cfg["vocab"], 3)
    want = O.model(cfg, W, toks)
    lost = O.model(cfg, W, toks[40:])
    for cuts in ([80], [40], [2], [1]):
        got = feed_all(eng, "a", toks, cuts)
        assert rel(got, want) < 5 * TOL and rel(got[40:], lost) > 0.05


def test_every_pass_of_a_loop_has_its_own_cache(tmp_path):
    cfg = config([gla(), parallel()], loop=(0, 2, 3))
    W = O.random_weights(cfg, seed=2, dtype=torch.float32)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    assert len(eng.kv_cache) == 6 and len({t.data_ptr() for l in eng.kv_cache for t in l}) == 9
    toks = tokens_of(50, cfg["vocab"], 1)
    once = copy.deepcopy(cfg)
    once["loop"]["times"] = 2
    shows(eng, cfg, W, (once, W), toks)
    del once["loop"]  # no loop at all
    assert rel(feed_all(load(once, W, tmp_path / "b", "cpu", torch.float32), "a", toks, [9, 1]), O.model(dict(once, loop={"start": 0, "stop": 0, "times": 1}), W, toks)) < TOL


def test_long_decoding(tmp_path):
    cfg = CASES["mixed"]
    W = slow(O.random_weights(cfg, seed=4, dtype=torch.float32), value=6.0)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    toks = tokens_of(250, cfg["vocab"], 1)
    want = O.model(cfg, {k: v.double() for k, v in W.items()}, toks)
    e = row_errors(feed_all(eng, "a", toks, [2, 1]), want)  # (a row whose state is almost nothing is normed up with its rounding)
    assert e.mean() < TOL and e.max() < 1e-3


# ------------------------------------------------------------------------------------------------ configuration, weights, command line
def test_configuration_round_trip_and_refusals(tmp_path):
    from miles_b200.models import ModelConfig, get_config

    for name, cfg in CASES.items():
        W = O.random_weights(cfg, rank=RANKS.get(name))
        mc = get_config(str(write_checkpoint(tmp_path / name, cfg, W)))  # (the decay's rank is read from the checkpoint's shapes)
        out = mc.to_hf_config()
        again = ModelConfig.from_hf_config(out)
        for l in out["layers"]:
            for m in (l["mixer"], l["mixer"].get("right", {})):
                m.pop("rank", None)
        assert out == cfg and mc.family == "pesanex" and again.plan == mc.plan
        n = sum(t.numel() for t in W.values())
        assert 0 <= mc.num_params() - n < 64 * len(cfg["layers"]) * 4 * cfg["width"]  # padding of fused weights only
    bad = [config([retention(decay=[0.5])]), config([parallel(heads=4, kv_heads=3)]), config([gla()], loop=(0, 2, 2)), config([retention(decay=[0.5, 1.5])])]
    for c in bad:
        with pytest.raises(ValueError):
            ModelConfig.from_hf_config(c)
    for c in (config([dict(gla(), type="other")]), config([dict(gla(), mlp={"kind": "routed", "ff": 8})]), config([retention(dims=3)])):
        with pytest.raises(NotImplementedError):
            ModelConfig.from_hf_config(c)


def test_weights_leave_under_checkpoint_names(tmp_path):
    from miles_b200.models.hf_mapping import hf_names, param_or_hf_view

    cfg = CASES["mixed"]
    W = O.random_weights(cfg, seed=3, dtype=torch.float32)
    eng = load(cfg, W, tmp_path, "cpu", torch.float32)
    out = dict(hf_names(eng.cfg, eng.store))
    assert set(out) == set(W) and all(torch.equal(out[k], W[k]) for k in W)
    param_or_hf_view(eng.cfg, eng.store, "l0.mix.left.k").zero_()  # a weight update under a checkpoint name
    assert dict(hf_names(eng.cfg, eng.store))["l0.mix.left.k"].abs().sum() == 0


def test_layout_description():
    from miles_b200.models import ModelConfig
    from miles_b200.models.cache_layout import cache_layout

    lay = cache_layout(ModelConfig.from_hf_config(CASES["mixed"]), torch.bfloat16)
    assert lay.has_state and len(lay.layers) == 6
    assert lay.bytes_per_slot() == 2 * (2 * (16 + 24) + 16 + 24)
    assert lay.bytes_per_sequence() == 4 * (2 * 2 * 16 * 24 + 2 * (2 * 40 * 24 + 3 * 24 * 16))


def test_trace_run_command(tmp_path):
    cfg = CASES["mixed"]
    W = O.random_weights(cfg, seed=11, dtype=torch.float32)
    d = write_checkpoint(tmp_path / "m", cfg, W)
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
    from miles_b200.utils.arguments import model_config_from_args, parse_args

    cfg = CASES["mixed"]
    W = O.random_weights(cfg, seed=3, dtype=torch.float32)
    d = write_checkpoint(tmp_path, cfg, W)
    engine, _, _ = build_from_args(["--hf-checkpoint", str(d), "--device", "cpu", "--max-running-requests", "2", "--page-size", "8",
                                    "--context-length", "64", "--max-prefill-tokens", "9"])
    toks = tokens_of(21, cfg["vocab"], 1)
    with TestClient(build_app(engine)) as client:
        r = client.post("/generate", json={"input_ids": toks, "sampling_params": {"temperature": 0.0, "max_new_tokens": 5}}).json()
    assert greedy_gap(cfg, W, toks, r["output_ids"]) < 1e-3
    with pytest.raises(NotImplementedError):
        model_config_from_args(parse_args(["--model-preset", "pesanex-smoke", "--num-rollout", "1", "--rollout-batch-size", "1"]))
