"""Kabadra without a GPU: configuration and checkpoint, the CPU executor through the engine against the plain oracle."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import kabadra_cases as kc
import kabadra_oracle as oracle

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 2e-5


def _want(cfg, w, toks):
    return oracle.forward(cfg, w, toks)[0]


# ------------------------------------------------------------------------------------------------ oracle and configuration
def test_sink_joins_the_denominator_only():
    s, sink = torch.tensor([0.3, -1.0, 2.0]), torch.tensor(0.7)
    full = torch.softmax(torch.cat([s, sink[None]]), 0)
    torch.testing.assert_close(oracle.sink_softmax(s, sink), full[:3])
    assert float(oracle.sink_softmax(s, torch.tensor(80.0)).sum()) < 1e-6


def test_window_keys_count_the_token_itself():
    assert oracle.window_keys(10, 3) == [8, 9, 10]
    assert oracle.window_keys(1, 3) == [0, 1]
    assert oracle.window_keys(7, 1) == [7]


def test_clamped_glu_limits_each_side():
    g, u = torch.tensor([[5.0, -9.0, 0.2]]), torch.tensor([[-7.0, 0.5, 9.0]])
    y = oracle.clamped_glu(torch.eye(3)[:1] * 0 + 1.0, torch.diag(g[0]), torch.diag(u[0]), torch.eye(3), 1.5)
    for i in range(3):
        a, b = min(float(g[0, i]), 1.5), max(-1.5, min(1.5, float(u[0, i])))
        assert abs(float(y[0, i]) - a / (1 + np.exp(-1.702 * a)) * (b + 1)) < 1e-6


def test_config_roundtrip_registry_and_validation(tmp_path):
    from tileinfer_b200.models import registry
    from tileinfer_b200.models.kabadra import KabadraConfig, KabadraWeights
    folder, cfg, w = kc.model(tmp_path, "mixed")
    mc = registry.config_from_dir(folder)
    assert isinstance(mc, KabadraConfig) and registry.family(mc.family).name == "kabadra"
    assert mc.to_dict() == cfg and mc.latent_owners == (0, 1) and mc.latent_layer(4) == 0
    assert mc.tensor_shapes() == oracle.tensor_shapes(cfg)
    src = KabadraWeights(mc, folder)
    assert all(torch.equal(src.get(n), w[n].float()) for n in w)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][2]["mixer"]["kv_from"] = 1                 # another rank
    with pytest.raises(ValueError):
        KabadraConfig.from_dict(bad)
    bad["layers"][2]["mixer"]["kv_from"] = 3                 # not an earlier layer with latents
    with pytest.raises(ValueError):
        KabadraConfig.from_dict(bad)
    with pytest.raises(ValueError):
        mc.validate_tp(2)
    assert "tiny-kabadra" in registry.all_presets() and "tiny-hybrid" in registry.all_presets()


def test_checkpoint_with_wrong_or_missing_tensor_is_refused(tmp_path):
    from tileinfer_b200.models.kabadra import KabadraConfig, KabadraWeights
    cfg = kc.ONE
    w = oracle.random_weights(cfg)
    less = {k: v for k, v in w.items() if k != "l0.mix.sink"}
    with pytest.raises(ValueError, match="sink"):
        KabadraWeights(KabadraConfig.from_dict(cfg), oracle.write_model(str(tmp_path / "a"), cfg, less))
    w["l0.mix.uk"] = w["l0.mix.uk"][:-1]
    with pytest.raises(ValueError, match="uk"):
        KabadraWeights(KabadraConfig.from_dict(cfg), oracle.write_model(str(tmp_path / "b"), cfg, w))


# ------------------------------------------------------------------------------------------------ CPU executor
@pytest.mark.parametrize("name", sorted(kc.CASES))
def test_whole_prompt_matches_oracle(tmp_path, name):
    folder, cfg, w = kc.model(tmp_path, name)
    t = kc.tokens(cfg, 90)
    got = kc.replay(kc.engine(folder, "bf16", "cpu"), [[("a", 90)]], {"a": t})["a"]
    assert kc.rms_error(got, _want(cfg, w, t)) < TOL


@pytest.mark.parametrize("sizes", [[1], [2], [3, 1, 16], [17, 15], [40, 1, 1]])
def test_portions_match_oracle(tmp_path, sizes):
    folder, cfg, w = kc.model(tmp_path, "mixed")
    t = kc.tokens(cfg, 83, seed=1)
    got = kc.replay(kc.engine(folder, "bf16", "cpu"), kc.cut("a", 83, sizes), {"a": t})["a"]
    assert kc.rms_error(got, _want(cfg, w, t)) < TOL


def test_batches_blocks_reused(tmp_path):
    folder, cfg, w = kc.model(tmp_path, "mixed")
    eng = kc.engine(folder, "bf16", "cpu", blocks=13)
    p = {r: kc.tokens(cfg, n, seed=n) for r, n in (("a", 70), ("b", 33), ("c", 9), ("d", 50), ("e", 21))}
    schedule = [[("a", 40), ("b", 2)], [("b", 1), ("c", 9), ("a", 2)], [("a", 28), ("b", 30)], [("d", 17), ("e", 20)],
                [("e", 1), ("d", 33)]]
    got = kc.replay(eng, schedule, p)
    for r, t in p.items():
        assert kc.rms_error(got[r], _want(cfg, w, t)) < TOL
    bm = eng.scheduler.block_manager
    assert bm.num_free_blocks == bm.num_blocks and len(eng.model_runner.free_deltanet_slots) == 4


def test_replay_refuses_what_does_not_fit(tmp_path):
    from tileinfer_b200.engine.replay import ReplaySession
    folder, cfg, _ = kc.model(tmp_path, "one")
    s = ReplaySession(kc.engine(folder, "bf16", "cpu", blocks=2, seqs=1))
    with pytest.raises(RuntimeError, match="blocks"):
        s.step([{"id": "a", "tokens": kc.tokens(cfg, 33), "want": []}])
    with pytest.raises(ValueError):
        ReplaySession(kc.engine(folder, "bf16", "cpu")).step([{"id": "a", "tokens": [cfg["vocab"]], "want": []}])


def _oracle_greedy(cfg, w, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(_want(cfg, w, t)[-1].argmax()))
    return t[len(prompt):]


@pytest.mark.parametrize("kw", [{}, {"max_prefill_chunk_tokens": 16, "num_scheduler_steps": 3},
                                {"blocks": 8, "swap_space_bytes": 1 << 20}, {"blocks": 8}])
def test_generation_through_the_scheduler(tmp_path, kw):
    """Greedy generation of several requests equals the oracle's, also with chunked prompts, and with too few blocks for
    all of them at once (swapped out or recomputed)."""
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = kc.model(tmp_path, "one")
    eng = kc.engine(folder, "bf16", "cpu", **{"blocks": 64, **kw})
    prompts = [kc.tokens(cfg, n, seed=n) for n in (30, 41, 18)]
    outs = eng.generate_token_ids(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True))
    assert outs == [_oracle_greedy(cfg, w, p, 24) for p in prompts]
    if kw.get("blocks") == 8:
        assert eng.scheduler.num_preemptions > 0


def test_prefix_reuse_needs_no_state(tmp_path):
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = kc.model(tmp_path, "one")
    eng = kc.engine(folder, "bf16", "cpu", enable_prefix_caching=True)
    base = kc.tokens(cfg, 50)
    sp = SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True)
    eng.generate_token_ids([base], sp)
    prompt = base[:40] + kc.tokens(cfg, 9, seed=5)
    assert eng.generate_token_ids([prompt], sp) == [_oracle_greedy(cfg, w, prompt, 5)]
    assert eng.scheduler.prefix_cache.hit_tokens == 32


def test_command_lines(tmp_path):
    """bin/trace_run and run_engine.py on a folder without tokenizer files and with a vocabulary too small for bytes."""
    cfg = kc.config([kc.layer(2, 16, 16, 24, 9, ff=32)], width=64, vocab=97)
    folder, cfg, w = kc.model(tmp_path, cfg)
    t = kc.tokens(cfg, 20)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": t[:13], "want": [0, 12]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": t[13:15], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": t[15:], "want": [4]}], "end": ["x"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "bfloat16", "--out", str(out),
                        "--max-tokens", "64", "--device", "cpu"], input="\n".join(map(json.dumps, lines)) + "\n",
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (out / "1.f32").exists()
    got = np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4") for i in (0, 2)]).reshape(3, -1)
    assert kc.rms_error(torch.from_numpy(got), _want(cfg, w, t)[[0, 12, 19]]) < TOL
    r = subprocess.run([sys.executable, os.path.join(ROOT, "run_engine.py"), "--model", folder, "--device", "cpu",
                        "--quantization", "bf16", "--prompt", " ".join(map(str, t)), "--max-tokens", "4", "--temperature", "0"],
                       capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.split()] == _oracle_greedy(cfg, w, t, 4)
