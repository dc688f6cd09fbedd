"""Luvapel without a GPU: the oracle's mechanisms, configuration and checkpoint, the CPU executor through the engine against the
plain oracle."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import luvapel_cases as lc
import luvapel_oracle as oracle

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 3e-5


def _want(cfg, w, toks):
    return oracle.forward(cfg, w, toks)[0]


# ------------------------------------------------------------------------------------------------ the oracle itself
def test_rotation_turns_neighbours_and_leaves_the_rest():
    x, pos = torch.randn(3, 2, 10), torch.tensor([0, 1, 7])
    y, a = oracle.rotate_pairs(x, pos, 100.0, 6), 7 * 100.0 ** (-4 / 6)      # pair 2 at position 7
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
    u, v, c, s = x[2, 1, 4], x[2, 1, 5], math.cos(a), math.sin(a)
    assert abs(float(y[2, 1, 4] - (u * c - v * s))) < 1e-5 and abs(float(y[2, 1, 5] - (v * c + u * s))) < 1e-5


def test_window_and_convolution():
    q, k, v = torch.zeros(5, 2), torch.zeros(5, 2), torch.arange(5.0)[:, None]
    assert oracle.windowed(q, k, v, 1.0, 3)[:, 0].tolist() == [0.0, 0.5, 1.0, 2.0, 3.0]
    u, w = torch.arange(1.0, 5.0)[:, None], torch.tensor([[100.0, 10.0, 1.0]])
    assert oracle.causal_conv(u, w)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0]


def test_values_are_keys_before_norm_and_rotation():
    """With a window of one token an attention head returns the key projection, whatever norm, rotation and temperature do."""
    m = lc.attention(2, 1, 6, 4, 1)
    g = torch.Generator().manual_seed(0)
    w = {n: torch.randn(s, generator=g) for n, s in (("q", (12, 5)), ("k", (6, 5)), ("q.norm", (6,)), ("k.norm", (6,)), ("temp", (2,)), ("g", (12, 5)), ("o", (5, 12)))}
    h = torch.randn(4, 5, generator=g)
    k = h @ w["k"].T
    want = (torch.cat([k, k], 1) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T
    torch.testing.assert_close(oracle.key_value_attention(h, w, m, "", 1e-5), want)


def test_delta_rule_replaces_what_a_key_holds():
    """Without decay and with full steps a unit key's read-out is the value written last; a decay scales what is old."""
    k = torch.eye(3)[[0, 1, 0]]
    v = torch.tensor([[1.0, 2.0], [3.0, 4.0], [5.0, 6.0]])
    o, S = oracle.delta_rule(k, k, v, torch.ones(3), torch.ones(3))
    assert torch.equal(o, v) and torch.equal(S, torch.tensor([[5.0, 6.0], [3.0, 4.0], [0.0, 0.0]]))
    _, S = oracle.delta_rule(k, k, v, torch.tensor([1.0, 0.5, 0.5]), torch.tensor([1.0, 1.0, 0.5]))
    assert torch.equal(S[1], 0.5 * v[1]) and torch.allclose(S[0], 0.25 * v[0] + 0.5 * (v[2] - 0.25 * v[0]))


def test_general_rule_reads_the_old_state():
    """Decay and removal both act on the state before the token; the key is written as projected."""
    r, k, v = torch.randn(5, 4), torch.randn(5, 4), torch.randn(5, 4)
    w, a = torch.rand(5, 4), torch.rand(5, 4)
    o, S = oracle.general_delta_rule(r, k, v, w, a)
    want = torch.zeros(4, 4)
    for t in range(5):
        u = k[t] / math.sqrt(float(k[t] @ k[t]) + 1e-6)
        want = (torch.diag(w[t]) - torch.outer(a[t] * u, u)) @ want + torch.outer(k[t], v[t])
        torch.testing.assert_close(o[t], want.T @ r[t])
    torch.testing.assert_close(S, want)
    o2, _ = oracle.general_delta_rule(r[3:], k[3:], v[3:], w[3:], a[3:], oracle.general_delta_rule(r[:3], k[:3], v[:3], w[:3], a[:3])[1])
    torch.testing.assert_close(o2, o[3:])


def test_gated_step_gates_before_the_norm():
    x, y = torch.randn(2, 4), torch.randn(2, 4)
    w = {"g": torch.zeros(4, 4), "g.b": torch.tensor([0.0, 50.0, -50.0, 0.0]), "n": torch.full((4,), 2.0)}
    z = y * torch.tensor([0.5, 1.0, 0.0, 0.5])
    want = x + 2 * z / (z.pow(2).mean(-1, keepdim=True) + 1e-6).sqrt()
    torch.testing.assert_close(oracle.gated_step(x, y, w, "g", "n", 1e-6), want)


# ------------------------------------------------------------------------------------------------ configuration, checkpoint
@pytest.mark.parametrize("name", sorted(lc.CASES))
def test_config_roundtrip_and_checkpoint(tmp_path, name):
    from tileinfer_b200.models import registry
    from tileinfer_b200.models.checkpoint import CheckpointWeights
    folder, cfg, w = lc.model(tmp_path, name)
    mc = registry.config_from_dir(folder)
    assert registry.family(mc.family).name == "luvapel" and mc.to_dict() == cfg and mc.recurrent
    assert mc.tensor_shapes() == {n: tuple(t.shape) for n, t in w.items()}
    src = CheckpointWeights(mc, folder)
    assert all(torch.equal(src.get(n), w[n].float()) for n in w)


def test_bad_configurations_are_refused():
    from tileinfer_b200.models.luvapel import LuvapelConfig
    good = json.dumps(lc.MIXED)

    def broken(change):
        d = json.loads(good)
        change(d["layers"], d)
        with pytest.raises((ValueError, KeyError)):
            LuvapelConfig.from_dict(d)
    broken(lambda e, d: e[0]["mixer"]["left"].update(kv_heads=4))                # heads do not divide
    broken(lambda e, d: e[0]["mixer"]["left"].update(vdim=41))                   # values are keys
    broken(lambda e, d: e[0]["mixer"]["left"]["rot"].update(dims=41))
    broken(lambda e, d: e[0]["mixer"]["left"]["mask"].update(size=0))
    broken(lambda e, d: e[0]["mixer"]["right"].update(kv_heads=5))
    broken(lambda e, d: e[0]["mixer"]["right"].update(conv=0))
    broken(lambda e, d: e[1]["mixer"].update(heads=0))
    broken(lambda e, d: e[0]["mlp"].update(kind="moe"))
    broken(lambda e, d: e[1].update(type="gla"))
    broken(lambda e, d: e[5].update(weights_of=7))                               # no such layer
    broken(lambda e, d: e[5].update(weights_of=6))                               # a layer without tensors of its own
    broken(lambda e, d: e[5].update(weights_of=0))                               # a layer that is not equal
    broken(lambda e, d: d.update(architecture="Nogidra"))
    with pytest.raises(ValueError):
        LuvapelConfig.from_dict(json.loads(good)).validate_tp(2)


def test_checkpoint_with_wrong_or_missing_tensor_is_refused(tmp_path):
    from tileinfer_b200.models.checkpoint import CheckpointWeights
    from tileinfer_b200.models.luvapel import LuvapelConfig
    mc, w = LuvapelConfig.from_dict(lc.ONE), oracle.random_weights(lc.ONE)
    less = {k: v for k, v in w.items() if k != "l0.mix.left.temp"}
    with pytest.raises(ValueError, match="left.temp"):
        CheckpointWeights(mc, oracle.write_model(str(tmp_path / "a"), lc.ONE, less))
    w["l0.mix.right.v.conv"] = w["l0.mix.right.v.conv"][:, 1:].contiguous()
    with pytest.raises(ValueError, match="v.conv"):
        CheckpointWeights(mc, oracle.write_model(str(tmp_path / "b"), lc.ONE, w))


def test_presets_and_random_weights():
    from tileinfer_b200.models import registry
    from tileinfer_b200.models.luvapel import TINY, make_weights
    assert {"tiny-luvapel", "luvapel-2k", "luvapel-4k"} <= set(registry.all_presets())
    a, b = make_weights(TINY, "random:1", None), make_weights(TINY, "random:1", None)
    assert torch.equal(a.get("l0.mix.right.v"), b.get("l0.mix.right.v")) and float(a.get("l1.norm2").min()) == 1.0


# ------------------------------------------------------------------------------------------------ CPU executor
@pytest.mark.parametrize("name", sorted(lc.CASES))
def test_whole_prompt_matches_oracle(tmp_path, name):
    folder, cfg, w = lc.model(tmp_path, name)
    t = lc.tokens(cfg, 70)
    got = lc.replay(lc.engine(folder, "bf16", "cpu"), [[("a", 70)]], {"a": t})["a"]
    assert lc.rms_error(got, _want(cfg, w, t)) < TOL


@pytest.mark.parametrize("sizes", [[1], [2], [3, 1, 16], [17, 15], [40, 1, 1]])
def test_portions_match_oracle(tmp_path, sizes):
    folder, cfg, w = lc.model(tmp_path, "mixed")
    t = lc.tokens(cfg, 67, seed=1)
    got = lc.replay(lc.engine(folder, "bf16", "cpu"), lc.cut("a", 67, sizes), {"a": t})["a"]
    assert lc.rms_error(got, _want(cfg, w, t)) < TOL


def test_batches_blocks_and_slots_reused(tmp_path):
    folder, cfg, w = lc.model(tmp_path, "mixed")
    eng = lc.engine(folder, "bf16", "cpu", blocks=13)
    p = {r: lc.tokens(cfg, n, seed=n) for r, n in (("a", 70), ("b", 33), ("c", 9), ("d", 50), ("e", 21))}
    schedule = [[("a", 40), ("b", 2)], [("b", 1), ("c", 9), ("a", 2)], [("a", 28), ("b", 30)], [("d", 17), ("e", 20)],
                [("e", 1), ("d", 33)]]
    got = lc.replay(eng, schedule, p)
    for r, t in p.items():
        assert lc.rms_error(got[r], _want(cfg, w, t)) < TOL
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
    folder, cfg, w = lc.model(tmp_path, "one")
    eng = lc.engine(folder, "bf16", "cpu", **{"blocks": 64, **kw})
    prompts = [lc.tokens(cfg, n, seed=n) for n in (30, 41, 18)]
    outs = eng.generate_token_ids(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))
    assert outs == [_oracle_greedy(cfg, w, p, 12) for p in prompts]
    if kw.get("blocks") == 7:
        assert eng.scheduler.num_preemptions > 0


@pytest.mark.parametrize("name", ["one", "recurrent"])
def test_prefix_reuse(tmp_path, name):
    """Cached pages, and the snapshot of states and convolution inputs."""
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = lc.model(tmp_path, name)
    eng = lc.engine(folder, "bf16", "cpu", enable_prefix_caching=True)
    base = lc.tokens(cfg, 50)
    sp = SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True)
    eng.generate_token_ids([base], sp)
    prompt = base[:49] + lc.tokens(cfg, 9, seed=5)
    assert eng.generate_token_ids([prompt], sp) == [_oracle_greedy(cfg, w, prompt, 5)]
    assert eng.scheduler.prefix_cache.hit_tokens == 48


def test_command_lines(tmp_path):
    """bin/trace_run and run_engine.py on a folder without tokenizer files and with a vocabulary too small for bytes."""
    folder, cfg, w = lc.model(tmp_path, "recurrent")
    t = lc.tokens(cfg, 20)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": t[:13], "want": [0, 12]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": t[13:15], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": t[15:], "want": [4]}], "end": ["x"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "bfloat16", "--out", str(out),
                        "--max-tokens", "64", "--device", "cpu"], input="\n".join(map(json.dumps, lines)) + "\n",
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4") for i in (0, 2)]).reshape(3, -1)
    assert lc.rms_error(torch.from_numpy(got), _want(cfg, w, t)[[0, 12, 19]]) < TOL
    r = subprocess.run([sys.executable, os.path.join(ROOT, "run_engine.py"), "--model", folder, "--device", "cpu",
                        "--quantization", "bf16", "--prompt", " ".join(map(str, t)), "--max-tokens", "4", "--temperature", "0"],
                       capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.split()] == _oracle_greedy(cfg, w, t, 4)
