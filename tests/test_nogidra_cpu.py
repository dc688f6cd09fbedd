"""Nogidra without a GPU: the oracle's mechanisms, configuration and checkpoint, the CPU executor through the engine against
the plain oracle."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import nogidra_cases as nc
import nogidra_oracle as oracle

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = 3e-5


def _want(cfg, w, toks):
    return oracle.forward(cfg, w, toks)[0]


# ------------------------------------------------------------------------------------------------ the oracle itself
def test_rotations_turn_their_pairs_and_leave_the_rest():
    x, pos = torch.randn(3, 2, 10), torch.tensor([0, 1, 7])
    a = 7 * 100.0 ** (-4 / 6)                               # pair 2 at position 7
    c, s = math.cos(a), math.sin(a)
    for rotate, (i, j) in ((oracle.rotate_halves, (2, 5)), (oracle.rotate_pairs, (4, 5))):
        y = rotate(x, pos, 100.0, 6)
        assert torch.equal(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
        u, v = x[2, 1, i], x[2, 1, j]
        assert abs(float(y[2, 1, i] - (u * c - v * s))) < 1e-5 and abs(float(y[2, 1, j] - (v * c + u * s))) < 1e-5


def test_windows_slopes_and_temperature():
    q, k, v = torch.zeros(5, 2), torch.zeros(5, 2), torch.arange(5.0)[:, None]
    assert oracle.windowed(q, k, v, 1.0, 3)[:, 0].tolist() == [0.0, 0.5, 1.0, 2.0, 3.0]
    two = oracle.windowed(q, k, v, 1.0, 2, slope=math.log(3.0))[4, 0]      # weights 3 : 1 for the token and the one before
    assert abs(float(two) - (0.75 * 4 + 0.25 * 3)) < 1e-6
    assert [oracle.slope(h, 4) for h in range(4)] == [0.25, 0.0625, 0.25 ** 3, 0.25 ** 4]
    assert [oracle.query_temperature(p, 2.0, 3) for p in (0, 1, 2, 4, 5)] == [1.0, 1.0, 1 + 2 * math.log(2), 1 + 2 * math.log(2), 1 + 2 * math.log(3)]


def test_convolution_looks_back():
    u, w = torch.arange(1.0, 5.0)[:, None], torch.tensor([[100.0, 10.0, 1.0]])
    assert oracle.causal_conv(u, w)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0]
    assert oracle.causal_conv(u, w, torch.tensor([0.5]))[0, 0] == 1.5


def test_state_space_is_the_decayed_sum():
    x, B, C, dt = torch.randn(6, 4), torch.randn(6, 3), torch.randn(6, 3), torch.rand(6)
    A, D = torch.tensor(0.3), torch.tensor(0.7)
    y, S = oracle.state_space(x, B, C, dt, A, D)
    for t in range(6):
        want = D * x[t]
        for j in range(t + 1):
            want = want + (C[t] @ B[j]) * dt[j] * torch.exp(-torch.exp(A) * dt[j + 1:t + 1].sum()) * x[j]
        torch.testing.assert_close(y[t], want, rtol=1e-4, atol=1e-5)
    y2, _ = oracle.state_space(x[4:], B[4:], C[4:], dt[4:], A, D, oracle.state_space(x[:4], B[:4], C[:4], dt[:4], A, D)[1])
    torch.testing.assert_close(y2, y[4:])


def test_group_norm_and_routing():
    y = torch.randn(2, 6)
    got = oracle.group_norm(y, torch.full((6,), 2.0), 3, 0.0)
    torch.testing.assert_close(got.view(2, 3, 2).pow(2).mean(-1), torch.full((2, 3), 4.0))
    ids, a = oracle.route(torch.ones(1, 1), torch.tensor([0.5, 2.0, -1.0, 1.0])[:, None], 2)
    assert ids.tolist() == [[1, 3]] and torch.allclose(a[0], torch.softmax(torch.tensor([2.0, 1.0]), 0))


# ------------------------------------------------------------------------------------------------ configuration, checkpoint
@pytest.mark.parametrize("name", sorted(nc.CASES))
def test_config_roundtrip_and_checkpoint(tmp_path, name):
    from tileinfer_b200.models import registry
    from tileinfer_b200.models.checkpoint import CheckpointWeights
    folder, cfg, w = nc.model(tmp_path, name)
    mc = registry.config_from_dir(folder)
    assert registry.family(mc.family).name == "nogidra" and mc.to_dict() == cfg and mc.recurrent == (name != "latent_only")
    assert mc.tensor_shapes() == {n: tuple(t.shape) for n, t in w.items()}
    src = CheckpointWeights(mc, folder)
    assert all(torch.equal(src.get(n), w[n].float()) for n in w)


def test_bad_configurations_are_refused():
    from tileinfer_b200.models.nogidra import NogidraConfig
    good = json.dumps(nc.MIXED)

    def broken(change):
        d = json.loads(good)
        change([e["mixer"] for e in d["layers"]], [e["mlp"] for e in d["layers"]], d)
        with pytest.raises((ValueError, KeyError)):
            NogidraConfig.from_dict(d)
    broken(lambda m, f, d: m[0]["left"].update(kv_heads=4))                      # heads do not divide
    broken(lambda m, f, d: m[0]["left"]["rot"].update(dims=41))
    broken(lambda m, f, d: m[0]["right"].update(groups=4))
    broken(lambda m, f, d: m[0]["right"].update(norm_groups=7))
    broken(lambda m, f, d: m[2]["rot"].update(dims=8))                           # part of the rotated part
    broken(lambda m, f, d: m[1]["mask"].update(size=0))
    broken(lambda m, f, d: m[1]["q_temp"].update(every=0))
    broken(lambda m, f, d: f[0]["router"].update(top=7))
    broken(lambda m, f, d: f[2].update(kind="sparse"))
    broken(lambda m, f, d: d["layers"][1].update(type="gla"))
    broken(lambda m, f, d: d.update(architecture="Kabadra"))
    with pytest.raises(ValueError):
        NogidraConfig.from_dict(json.loads(good)).validate_tp(2)


def test_checkpoint_with_wrong_or_missing_tensor_is_refused(tmp_path):
    from tileinfer_b200.models.checkpoint import CheckpointWeights
    from tileinfer_b200.models.nogidra import NogidraConfig
    mc, w = NogidraConfig.from_dict(nc.ONE), oracle.random_weights(nc.ONE)
    less = {k: v for k, v in w.items() if k != "l0.mix.left.k.b"}
    with pytest.raises(ValueError, match="left.k.b"):
        CheckpointWeights(mc, oracle.write_model(str(tmp_path / "a"), nc.ONE, less))
    w["l1.mix.v.conv"] = w["l1.mix.v.conv"][:, 1:].contiguous()
    with pytest.raises(ValueError, match="v.conv"):
        CheckpointWeights(mc, oracle.write_model(str(tmp_path / "b"), nc.ONE, w))


def test_presets_and_random_weights():
    from tileinfer_b200.models import registry
    from tileinfer_b200.models.nogidra import TINY, make_weights
    assert {"tiny-nogidra", "nogidra-2k", "nogidra-4k"} <= set(registry.all_presets())
    a, b = make_weights(TINY, "random:1", None), make_weights(TINY, "random:1", None)
    assert torch.equal(a.get("l0.mix.right.in"), b.get("l0.mix.right.in"))
    assert not a.get("l0.norm1").any() and not a.get("final.norm").any() and float(a.get("l2.mix.dkv.norm").min()) == 1.0


# ------------------------------------------------------------------------------------------------ CPU executor
@pytest.mark.parametrize("name", sorted(nc.CASES))
def test_whole_prompt_matches_oracle(tmp_path, name):
    folder, cfg, w = nc.model(tmp_path, name)
    t = nc.tokens(cfg, 70)
    got = nc.replay(nc.engine(folder, "bf16", "cpu"), [[("a", 70)]], {"a": t})["a"]
    assert nc.rms_error(got, _want(cfg, w, t)) < TOL


@pytest.mark.parametrize("sizes", [[1], [2], [3, 1, 16], [17, 15], [40, 1, 1]])
def test_portions_match_oracle(tmp_path, sizes):
    folder, cfg, w = nc.model(tmp_path, "mixed")
    t = nc.tokens(cfg, 67, seed=1)
    got = nc.replay(nc.engine(folder, "bf16", "cpu"), nc.cut("a", 67, sizes), {"a": t})["a"]
    assert nc.rms_error(got, _want(cfg, w, t)) < TOL


def test_batches_blocks_and_slots_reused(tmp_path):
    folder, cfg, w = nc.model(tmp_path, "mixed")
    eng = nc.engine(folder, "bf16", "cpu", blocks=13)
    p = {r: nc.tokens(cfg, n, seed=n) for r, n in (("a", 70), ("b", 33), ("c", 9), ("d", 50), ("e", 21))}
    schedule = [[("a", 40), ("b", 2)], [("b", 1), ("c", 9), ("a", 2)], [("a", 28), ("b", 30)], [("d", 17), ("e", 20)],
                [("e", 1), ("d", 33)]]
    got = nc.replay(eng, schedule, p)
    for r, t in p.items():
        assert nc.rms_error(got[r], _want(cfg, w, t)) < TOL
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
    folder, cfg, w = nc.model(tmp_path, "one")
    eng = nc.engine(folder, "bf16", "cpu", **{"blocks": 64, **kw})
    prompts = [nc.tokens(cfg, n, seed=n) for n in (30, 41, 18)]
    outs = eng.generate_token_ids(prompts, SamplingParams(temperature=0.0, max_tokens=16, ignore_eos=True))
    assert outs == [_oracle_greedy(cfg, w, p, 16) for p in prompts]
    if kw.get("blocks") == 7:
        assert eng.scheduler.num_preemptions > 0


@pytest.mark.parametrize("name", ["one", "latent_only"])
def test_prefix_reuse(tmp_path, name):
    """Cached pages, and for recurrent models the snapshot of states and convolution inputs."""
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = nc.model(tmp_path, name)
    eng = nc.engine(folder, "bf16", "cpu", enable_prefix_caching=True)
    base = nc.tokens(cfg, 50)
    sp = SamplingParams(temperature=0.0, max_tokens=5, ignore_eos=True)
    eng.generate_token_ids([base], sp)
    prompt = base[:49] + nc.tokens(cfg, 9, seed=5)
    assert eng.generate_token_ids([prompt], sp) == [_oracle_greedy(cfg, w, prompt, 5)]
    assert eng.scheduler.prefix_cache.hit_tokens == 48


def test_command_lines(tmp_path):
    """bin/trace_run and run_engine.py on a folder without tokenizer files and with a vocabulary too small for bytes."""
    folder, cfg, w = nc.model(tmp_path, "latent_only")
    t = nc.tokens(cfg, 20)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": t[:13], "want": [0, 12]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": t[13:15], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": t[15:], "want": [4]}], "end": ["x"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "bfloat16", "--out", str(out),
                        "--max-tokens", "64", "--device", "cpu"], input="\n".join(map(json.dumps, lines)) + "\n",
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4") for i in (0, 2)]).reshape(3, -1)
    assert nc.rms_error(torch.from_numpy(got), _want(cfg, w, t)[[0, 12, 19]]) < TOL
    r = subprocess.run([sys.executable, os.path.join(ROOT, "run_engine.py"), "--model", folder, "--device", "cpu",
                        "--quantization", "bf16", "--prompt", " ".join(map(str, t)), "--max-tokens", "4", "--temperature", "0"],
                       capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.split()] == _oracle_greedy(cfg, w, t, 4)


# ------------------------------------------------------------------------------------------------ work lists of the kernels
def test_convolution_tiles_cover_every_token_once():
    from tileinfer_b200.ops.functional import CONV_TILE, conv_tiles
    seq, tok, n = conv_tiles([0, 1, 1 + CONV_TILE, 40 + CONV_TILE]).tolist()
    assert sum(n) == 40 + CONV_TILE and max(n) <= CONV_TILE and seq == sorted(seq)
    assert [a + b for a, b in zip(tok, n)] == tok[1:] + [40 + CONV_TILE]
