"""Gerivik without a GPU: the oracle's mechanisms, configuration and checkpoint, the CPU executor through the engine
against the plain oracle."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import gerivik_cases as gc
import gerivik_oracle as oracle

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 3e-5


def _want(cfg, w, toks):
    return oracle.forward(cfg, w, toks)[0]


# ------------------------------------------------------------------------------------------------ the oracle itself
def test_rotation_turns_pairs_and_leaves_the_rest():
    x = torch.randn(3, 2, 10)
    y = oracle.rotate(x, torch.tensor([0, 1, 7]), 100.0, 6)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
    a = 7 * 100.0 ** (-4 / 6)                               # pair (2, 5) at position 7
    assert abs(float(y[2, 1, 2]) - float(x[2, 1, 2] * math.cos(a) - x[2, 1, 5] * math.sin(a))) < 1e-5
    assert abs(float(y[2, 1, 5]) - float(x[2, 1, 5] * math.cos(a) + x[2, 1, 2] * math.sin(a))) < 1e-5


def test_recurrence_is_the_decayed_sum():
    q, k, v = torch.randn(5, 3), torch.randn(5, 3), torch.randn(5, 4)
    alpha = torch.rand(5, 3)
    o, S = oracle.recurrence(q, k, v, alpha)
    for t in range(5):
        want = torch.zeros(4)
        for j in range(t + 1):
            want += (q[t] * k[j] * alpha[j + 1:t + 1].prod(0)).sum() * v[j]
        torch.testing.assert_close(o[t], want, rtol=1e-4, atol=1e-5)
    o2, _ = oracle.recurrence(q[3:], k[3:], v[3:], alpha[3:], oracle.recurrence(q[:3], k[:3], v[:3], alpha[:3])[1])
    torch.testing.assert_close(o2, o[3:])


def test_routing_uses_groups_corrections_and_plain_weights():
    r = {"experts": 4, "identity": 2, "top": 2, "groups": {"count": 3, "keep": 1}}
    w = torch.tensor([2.0, 1.0, 0.0, 0.0, 0.5, 0.4])[:, None]
    s = torch.softmax(w[:, 0], 0)
    ids, a = oracle.route(torch.ones(1, 1), w, torch.zeros(6), r)
    assert ids.tolist() == [[0, 1]] and torch.allclose(a[0], s[:2])
    # corrections move the choice (all negative here: left-out experts must not beat them) but not the weights
    ids, a = oracle.route(torch.ones(1, 1), w, torch.tensor([-3.0, -3.0, -2.0, -2.5, -1.0, -1.2]), r)
    assert ids.tolist() == [[4, 5]] and torch.allclose(a[0], s[4:])


def test_capped_scores():
    s = torch.tensor([0.01, -2.0, 50.0])
    torch.testing.assert_close(oracle.capped(s, 3.0), torch.tensor([0.01, -3 * math.tanh(2 / 3), 3.0]), rtol=1e-5, atol=1e-6)


# ------------------------------------------------------------------------------------------------ configuration, checkpoint
@pytest.mark.parametrize("name", sorted(gc.CASES))
def test_config_roundtrip_and_checkpoint(tmp_path, name):
    from tileinfer_b200.models import registry
    from tileinfer_b200.models.checkpoint import CheckpointWeights
    folder, cfg, w = gc.model(tmp_path, name)
    mc = registry.config_from_dir(folder)
    assert registry.family(mc.family).name == "gerivik" and mc.to_dict() == cfg and mc.recurrent
    assert mc.tensor_shapes() == {n: tuple(t.shape) for n, t in w.items()}       # the decay's rank comes from the tensors
    src = CheckpointWeights(mc, folder)
    assert all(torch.equal(src.get(n), w[n].float()) for n in w)


def test_bad_configurations_are_refused():
    from tileinfer_b200.models.gerivik import GerivikConfig
    good = json.dumps(gc.MIXED)

    def broken(change):
        d = json.loads(good)
        change(d)
        with pytest.raises((ValueError, KeyError)):
            GerivikConfig.from_dict(d)
    broken(lambda d: d["layers"][4].update(weights_of=5))                        # a layer without tensors
    broken(lambda d: d["layers"][4]["mixer"].update(tau=4.0))                    # not equal to its owner
    broken(lambda d: d["layers"][1]["mixer"].update(kv_heads=4))                 # heads do not divide
    broken(lambda d: d["layers"][1]["mixer"]["rot"].update(dims=41))
    broken(lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=3))
    broken(lambda d: d["layers"][3]["mlp"]["router"].update(top=4))              # more than the kept groups hold
    broken(lambda d: d["layers"][0].update(type="mamba"))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="dense"))
    with pytest.raises(ValueError):
        GerivikConfig.from_dict(json.loads(good)).validate_tp(2)


def test_checkpoint_with_wrong_or_missing_tensor_is_refused(tmp_path):
    from tileinfer_b200.models.checkpoint import CheckpointWeights
    from tileinfer_b200.models.gerivik import GerivikConfig
    mc, w = GerivikConfig.from_dict(gc.ONE, decay_rank={0: 8}), oracle.random_weights(gc.ONE)
    less = {k: v for k, v in w.items() if k != "l1.mlp.e3.up"}
    with pytest.raises(ValueError, match="e3.up"):
        CheckpointWeights(mc, oracle.write_model(str(tmp_path / "a"), gc.ONE, less))
    w["l0.mix.a2"] = w["l0.mix.a2"][:-1]
    with pytest.raises(ValueError, match="a2"):
        CheckpointWeights(mc, oracle.write_model(str(tmp_path / "b"), gc.ONE, w))


def test_presets_and_random_weights():
    from tileinfer_b200.models import registry
    from tileinfer_b200.models.gerivik import TINY, make_weights
    assert {"tiny-gerivik", "gerivik-2k", "gerivik-4k"} <= set(registry.all_presets())
    a, b = make_weights(TINY, "random:1", None), make_weights(TINY, "random:1", None)
    assert torch.equal(a.get("l0.mix.a2"), b.get("l0.mix.a2")) and float(a.get("l0.norm1b").min()) == 1.0
    assert TINY.owner(5) == 1 and TINY.layers[5].weights_of == 1


# ------------------------------------------------------------------------------------------------ CPU executor
@pytest.mark.parametrize("name", sorted(gc.CASES))
def test_whole_prompt_matches_oracle(tmp_path, name):
    folder, cfg, w = gc.model(tmp_path, name)
    t = gc.tokens(cfg, 70)
    got = gc.replay(gc.engine(folder, "bf16", "cpu"), [[("a", 70)]], {"a": t})["a"]
    assert gc.rms_error(got, _want(cfg, w, t)) < TOL


@pytest.mark.parametrize("sizes", [[1], [2], [3, 1, 16], [17, 15], [40, 1, 1]])
def test_portions_match_oracle(tmp_path, sizes):
    folder, cfg, w = gc.model(tmp_path, "mixed")
    t = gc.tokens(cfg, 67, seed=1)
    got = gc.replay(gc.engine(folder, "bf16", "cpu"), gc.cut("a", 67, sizes), {"a": t})["a"]
    assert gc.rms_error(got, _want(cfg, w, t)) < TOL


def test_batches_blocks_and_slots_reused(tmp_path):
    folder, cfg, w = gc.model(tmp_path, "mixed")
    eng = gc.engine(folder, "bf16", "cpu", blocks=13)
    p = {r: gc.tokens(cfg, n, seed=n) for r, n in (("a", 70), ("b", 33), ("c", 9), ("d", 50), ("e", 21))}
    schedule = [[("a", 40), ("b", 2)], [("b", 1), ("c", 9), ("a", 2)], [("a", 28), ("b", 30)], [("d", 17), ("e", 20)],
                [("e", 1), ("d", 33)]]
    got = gc.replay(eng, schedule, p)
    for r, t in p.items():
        assert gc.rms_error(got[r], _want(cfg, w, t)) < TOL
    bm = eng.scheduler.block_manager
    assert bm.num_free_blocks == bm.num_blocks and len(eng.model_runner.free_deltanet_slots) == 4


def _oracle_greedy(cfg, w, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(_want(cfg, w, t)[-1].argmax()))
    return t[len(prompt):]


@pytest.mark.parametrize("kw", [{}, {"max_prefill_chunk_tokens": 16, "num_scheduler_steps": 3},
                                {"blocks": 7, "swap_space_bytes": 1 << 20}, {"blocks": 7}])
def test_generation_through_the_scheduler(tmp_path, kw):
    """Greedy generation of several requests equals the oracle's, also with chunked prompts, and with too few blocks for
    all of them at once (swapped out with their states, or recomputed)."""
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = gc.model(tmp_path, "one")
    eng = gc.engine(folder, "bf16", "cpu", **{"blocks": 64, **kw})
    prompts = [gc.tokens(cfg, n, seed=n) for n in (30, 41, 18)]
    outs = eng.generate_token_ids(prompts, SamplingParams(temperature=0.0, max_tokens=16, ignore_eos=True))
    assert outs == [_oracle_greedy(cfg, w, p, 16) for p in prompts]
    if kw.get("blocks") == 7:
        assert eng.scheduler.num_preemptions > 0


def test_prefix_reuse_restores_the_state(tmp_path):
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = gc.model(tmp_path, "one")
    eng = gc.engine(folder, "bf16", "cpu", enable_prefix_caching=True)
    base = gc.tokens(cfg, 50)
    sp = SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True)
    eng.generate_token_ids([base], sp)
    prompt = base[:49] + gc.tokens(cfg, 9, seed=5)
    assert eng.generate_token_ids([prompt], sp) == [_oracle_greedy(cfg, w, prompt, 5)]
    assert eng.scheduler.prefix_cache.hit_tokens == 48


def test_command_lines(tmp_path):
    """bin/trace_run and run_engine.py on a folder without tokenizer files and with a vocabulary too small for bytes."""
    folder, cfg, w = gc.model(tmp_path, "state_only")
    t = gc.tokens(cfg, 20)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": t[:13], "want": [0, 12]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": t[13:15], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": t[15:], "want": [4]}], "end": ["x"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "bfloat16", "--out", str(out),
                        "--max-tokens", "64", "--device", "cpu"], input="\n".join(map(json.dumps, lines)) + "\n",
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    got = np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4") for i in (0, 2)]).reshape(3, -1)
    assert gc.rms_error(torch.from_numpy(got), _want(cfg, w, t)[[0, 12, 19]]) < TOL
    r = subprocess.run([sys.executable, os.path.join(ROOT, "run_engine.py"), "--model", folder, "--device", "cpu",
                        "--quantization", "bf16", "--prompt", " ".join(map(str, t)), "--max-tokens", "4", "--temperature", "0"],
                       capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.split()] == _oracle_greedy(cfg, w, t, 4)


# ------------------------------------------------------------------------------------------------ work lists of the kernels
def test_chunk_table_cuts_at_chunks_and_snapshot_points():
    from tileinfer_b200.ops.functional import gla_chunk_table
    ck, rng = gla_chunk_table([0, 5, 150, 190], [1, 2], 64, [{}, {48: 0, 112: 1}, {}])
    assert rng.tolist() == [0, 3, 4]
    assert ck.tolist() == [[1, 1, 1, 2], [5, 53, 117, 150], [48, 64, 33, 40], [0, 1, -1, -1]]
