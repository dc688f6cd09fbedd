"""Kabadra on the GPU: each kernel against plain PyTorch fp32, the model against the plain oracle in every precision, and
the engine (portions, batches, reused pages, long decoding, generation)."""
import json
import math
import os
import subprocess

import numpy as np
import pytest
import torch

import kabadra_cases as kc
import kabadra_oracle as oracle

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = torch.bfloat16, torch.float32
# largest error of a position's logits relative to the size of the logits
TOL = {"bf16": 0.03, "fp32": 1e-4, "w8a16": 0.03}


@pytest.fixture(scope="module")
def F():
    from tileinfer_b200.ops import functional
    functional.L("base", "rows", "latent")
    return functional


def rel(got, want):
    return ((got.float() - want.float()).norm() / want.float().norm().clamp_min(1e-20)).item()


def _rows(t, pitch):
    out = torch.zeros(t.shape[0], pitch, dtype=t.dtype, device=t.device)
    out[:, :t.shape[1]] = t
    return out


# ------------------------------------------------------------------------------------------------ row operations
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("W", [40, 136, 2056, 9000])
def test_embedding_with_positions_and_norms(F, dtype, W):
    P, V, T = -(-W // 64) * 64, 77, 9
    g = torch.Generator().manual_seed(0)
    e, p = (torch.randn(n, W, generator=g).to(dtype).cuda() for n in (V, 50))
    w = (torch.rand(W, generator=g) + 0.5).cuda()
    ids, pos = torch.randint(0, V, (T,), generator=g).cuda(), torch.randint(0, 50, (T,), generator=g).int().cuda()
    x = torch.full((T, P), 7.0, device="cuda")
    F.embed_pos(ids, pos, _rows(e, P), _rows(p, P), _rows(w[None], P)[0], x, W, 1e-3)
    want = oracle.rms_norm(e[ids].float() + p[pos.long()].float(), w, 1e-3)
    assert rel(x[:, :W], want) < 1e-6 and not x[:, W:].any()
    y = torch.full((T, P), 7.0, dtype=dtype, device="cuda")
    F.rmsnorm_f32(x, _rows(w[None], P)[0], y, W, 1e-3)
    assert rel(y[:, :W], oracle.rms_norm(x[:, :W], w, 1e-3)) < (1e-6 if dtype == F32 else 4e-3) and not y[:, W:].any()
    F.embed_pos(ids, pos, _rows(e, P), None, None, x, W, 1e-3)            # neither positions nor norm
    assert torch.equal(x[:, :W], e[ids].float())


@pytest.mark.parametrize("dtype", [BF16, F32])
def test_latent_store_and_gather(F, dtype):
    T, R, Rp, col, nb = 11, 72, 128, 64, 4
    proj = torch.zeros(T, 64 + Rp + 8, dtype=dtype, device="cuda")
    proj[:, col:col + R] = torch.randn(T, R, device="cuda").to(dtype)
    w = torch.zeros(Rp, device="cuda")
    w[:R] = torch.rand(R, device="cuda") + 0.5
    cache = torch.zeros(nb, 16, Rp, dtype=dtype, device="cuda")
    slots = torch.tensor([5, 16, -1, 63, 40, 0, 1, 2, 64, 33, 17], device="cuda")       # -1 and 64: not in the cache
    F.latent_store(proj, col, w, slots, cache, R, 1e-4)
    want = torch.zeros_like(cache).view(-1, Rp)
    ok = (slots >= 0) & (slots < nb * 16)
    want[slots[ok], :R] = oracle.rms_norm(proj[:, col:col + R].float(), w[:R], 1e-4)[ok].to(dtype)
    assert rel(cache.view(-1, Rp), want) < (1e-6 if dtype == F32 else 3e-3)
    out = torch.full((T, Rp), 9.0, dtype=dtype, device="cuda")
    F.latent_gather(cache, slots, out)
    assert torch.equal(out[ok], cache.view(-1, Rp)[slots[ok]]) and not out[~ok].any()


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("M,H,N,K", [(1, 3, 64, 64), (17, 5, 128, 64), (40, 2, 64, 192)])
def test_head_product(F, dtype, M, H, N, K):
    ld, gcol = H * K + 16, H * K + 3
    x = torch.randn(M, ld, device="cuda").to(dtype)
    w = (torch.randn(H, N, K, device="cuda") / math.sqrt(K)).to(dtype)
    out = torch.zeros(M, H * N + 64, dtype=dtype, device="cuda")
    F.head_product(x, w, out, gate=x, gcol=gcol)
    want = torch.einsum("mhk,hnk->mhn", x[:, :H * K].float().view(M, H, K), w.float())
    tol = 1e-5 if dtype == F32 else 4e-3
    assert rel(out[:, :H * N].view(M, H, N), want * torch.sigmoid(x[:, gcol:gcol + H].float())[..., None]) < tol
    assert not out[:, H * N:].any()
    F.head_product(x, w, out)
    assert rel(out[:, :H * N].view(M, H, N), want) < tol


# M covers the token tiles; K = 6144 with few rows is cut along k
@pytest.mark.parametrize("kind", ["bf16", "w8a16", "fp32"])
@pytest.mark.parametrize("M,N,K", [(1, 128, 64), (5, 264, 192), (40, 136, 6144), (200, 1032, 320), (3, 2560, 4096)])
def test_product_epilogues(F, kind, M, N, K):
    from tileinfer_b200.models.latent_b200 import Product
    torch.manual_seed(M)
    dt = F32 if kind == "fp32" else BF16
    w = torch.randn(N, K, device="cuda") / math.sqrt(K)
    x = torch.randn(M, K, device="cuda").to(dt)
    p = Product(w, kind, "cuda")
    wf = kc.quantised({"a.q": w})["a.q"] if kind == "w8a16" else w.to(dt)
    y = x.float().double() @ wf.double().t()
    # fp32 residual, in place
    r = torch.randn(M, N, device="cuda")
    out = r.clone()
    p(x, out, F.GEPI_RESID32, F.gemm_epilogue(resid32=out))
    assert (out.double() - r.double() - y).abs().max() < (1e-4 if kind != "w8a16" else 4e-3)
    # scaled fp32 (vocabulary product)
    out = torch.empty(M, N, device="cuda")
    p(x, out, F.GEPI_F32, F.gemm_epilogue(scale=0.37))
    assert rel(out, 0.37 * y) < (1e-5 if kind != "w8a16" else 1e-3)
    # stored rows, then (gate, up) pairs through the clamped unit; most values are beyond the limit
    ns = 64
    a, b = torch.zeros(M, ns, dtype=dt, device="cuda"), torch.zeros(M, (N - ns) // 2 + 4, dtype=dt, device="cuda")
    p(x, a, F.GEPI_SPLIT_GLU, F.gemm_epilogue(out2=b[:, :(N - ns) // 2], n_split=ns, glu=(0.4, 1.702, 1.0)))
    gate, up = y[:, ns::2].clamp(max=0.4), y[:, ns + 1::2].clamp(-0.4, 0.4)
    tol = 2e-5 if kind == "fp32" else 6e-3
    assert rel(a, y[:, :ns]) < tol and rel(b[:, :(N - ns) // 2], gate * torch.sigmoid(1.702 * gate) * (up + 1.0)) < tol
    assert not b[:, (N - ns) // 2:].any()


# ------------------------------------------------------------------------------------------------ attention kernels
def _attn_ref(q, c, pos, window, scale, sink):
    """q [T, H, R], c [n, R] (position = row), pos [T]."""
    s = torch.einsum("thr,nr->htn", q.float(), c.float()) * scale
    d = pos[:, None] - torch.arange(c.shape[0], device=c.device)[None]
    out = (d < 0) | ((d >= window) if window else torch.zeros_like(d, dtype=torch.bool))
    s = s.masked_fill(out[None], float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink[:, None, None].expand(-1, s.shape[1], 1)], -1)
    a = torch.softmax(s, -1)[..., :c.shape[0]]
    return torch.einsum("htn,nr->thr", a, c.float())


def _paged(c, seed=0):
    """Latents [n, R] of one sequence in shuffled pages of a larger cache; the free pages hold large values."""
    n, R = c.shape
    nb = -(-n // 16)
    g = torch.Generator().manual_seed(seed)
    table = torch.randperm(nb + 5, generator=g)[:nb]
    cache = torch.full((nb + 5, 16, R), 50.0, dtype=c.dtype, device="cuda")
    full = torch.full((nb * 16, R), 50.0, dtype=c.dtype, device="cuda")       # the tail of the last page too
    full[:n] = c
    cache[table.cuda()] = full.view(nb, 16, R)
    return cache, table.int().cuda()[None]


def _run_latent_attn(F, q, cache, table, pos, window, scale, sink, nsplit):
    T, H, R = q.shape
    rows = 32 if H > 16 else 16
    part = torch.empty(T * -(-H // rows) * nsplit * rows * R, device="cuda")
    ml = torch.empty(part.numel() // R * 2, device="cuda")
    idx, one, zero = torch.arange(T, dtype=torch.int32, device="cuda"), torch.ones(T, dtype=torch.int32, device="cuda"), \
        torch.zeros(T, dtype=torch.int32, device="cuda")
    out = torch.zeros_like(q)
    p = F.LatentAttnParams()
    p.q, p.cache, p.out, p.sink = q.data_ptr(), cache.data_ptr(), out.data_ptr(), 0 if sink is None else sink.data_ptr()
    p.block_tables, p.positions = table.data_ptr(), pos.data_ptr()
    p.qg_seq, p.qg_tok0, p.qg_ntok = zero.data_ptr(), idx.data_ptr(), one.data_ptr()
    p.o_part, p.ml_part = part.data_ptr(), ml.data_ptr()
    p.H, p.R, p.Rp, p.max_blocks, p.nsplit, p.num_qg = H, R, R, table.shape[1], nsplit, T
    p.window, p.num_blocks, p.scale = window, cache.shape[0], scale
    F.latent_attn(p, q.dtype == F32)
    torch.cuda.synchronize()
    return out


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,R,window,nsplit", [(1, 64, 0, 1), (4, 128, 50, 3), (16, 192, 129, 1), (17, 256, 64, 2), (40, 320, 200, 4),
                                               (5, 384, 1, 1), (33, 448, 77, 1), (3, 512, 0, 5), (32, 512, 300, 32), (2, 640, 90, 1)])
def test_latent_attention(F, dtype, H, R, window, nsplit):
    torch.manual_seed(R + H)
    n = 411
    c = torch.randn(n, R, device="cuda").to(dtype)
    cache, table = _paged(c)
    pos = torch.tensor([0, 1, 15, 16, 63, 64, 130, 255, 256, 400, 410], dtype=torch.int32, device="cuda")
    q = torch.randn(len(pos), H, R, device="cuda").to(dtype)
    for sink in (torch.randn(H, device="cuda") * 2, None):
        out = _run_latent_attn(F, q, cache, table, pos, window, 2.0 / math.sqrt(R), sink, nsplit)
        want = _attn_ref(q, c, pos.long(), window, 2.0 / math.sqrt(R), sink)
        assert rel(out, want) < (2e-5 if dtype == F32 else 6e-3)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("R,window,nsplit", [(64, 33, 1), (128, 100, 2), (512, 200, 3), (512, 16, 1)])
def test_latent_attention_window_edge(F, dtype, R, window, nsplit):
    """One key carries all the weight: the query sees it while it is window - 1 tokens back, and no longer one token on."""
    for key in (0, 15, 16, 47, 128):
        c = torch.randn(key + window + 40, R, device="cuda") * 0.1
        c[:, 0] = 0
        c[key] = 0
        c[key, 0], c[key, 1] = 1.0, 5.0
        c = c.to(dtype)
        cache, table = _paged(c, seed=key)
        pos = torch.tensor([key, key + 1, key + window - 1, key + window, key + window + 1], dtype=torch.int32, device="cuda")
        q = torch.zeros(len(pos), 3, R, device="cuda")
        q[:, :, 0] = 40.0
        out = _run_latent_attn(F, q.to(dtype), cache, table, pos, window, 1.0, torch.zeros(3, device="cuda"), nsplit)
        assert (out[:3, :, 1] - 5.0).abs().max() < 0.05
        assert out[3:, :, 1].abs().max() < 1.0


def test_latent_attention_sink_takes_its_share(F):
    """Equal scores: with a sink of log(n) the keys keep exactly half of the weight, in one split or several."""
    n, R = 200, 128
    c = torch.zeros(n, R, device="cuda")
    c[:, 1] = 2.0
    cache, table = _paged(c.to(BF16))
    q, pos = torch.zeros(1, 20, R, dtype=BF16, device="cuda"), torch.tensor([n - 1], dtype=torch.int32, device="cuda")
    for nsplit in (1, 4):
        out = _run_latent_attn(F, q, cache, table, pos, 0, 1.0, torch.full((20,), math.log(n), device="cuda"), nsplit)
        assert (out[..., 1] - 1.0).abs().max() < 1e-2


def _prefill(F, q, k, v, pos0, lo, window, scale, sink, gate):
    """q [T, H, dp]; k, v rows from position lo on."""
    T, H, dp = q.shape
    vp = v.shape[-1]
    proj = torch.cat([q.flatten(1), gate, torch.zeros(T, -H % 8, dtype=BF16, device="cuda")], 1).contiguous()
    pad = torch.full((3, H * (dp + vp)), 30.0, dtype=BF16, device="cuda")            # rows of some other sequence around
    kv = torch.cat([pad, torch.cat([k.flatten(1), v.flatten(1)], 1), pad]).contiguous()
    tiles = torch.tensor([(a, min(128, T - a), pos0 + a, 3, lo) for a in range(0, T, 128)], dtype=torch.int32).t().contiguous().cuda()
    out = torch.zeros(T, H * vp + 8, dtype=BF16, device="cuda")
    F.latent_prefill(proj, kv, tiles, out, H=H, dp=dp, vp=vp, window=window, scale=scale, sink=sink, gate=proj, gcol=H * dp)
    torch.cuda.synchronize()
    assert not out[:, H * vp:].any()
    return out[:, :H * vp].view(T, H, vp)


@pytest.mark.parametrize("H,dp,vp,window,start,T", [(2, 64, 64, 50, 0, 40), (3, 64, 128, 72, 100, 200), (2, 128, 128, 0, 0, 300),
                                                    (3, 128, 64, 128, 777, 513), (2, 192, 128, 129, 64, 130), (1, 256, 256, 1000, 500, 700),
                                                    (2, 64, 192, 1, 5, 129), (1, 256, 64, 33, 0, 128), (1, 64, 256, 257, 256, 33)])
def test_prefill_attention(F, H, dp, vp, window, start, T):
    torch.manual_seed(T)
    lo = max(0, start - window + 1) if window else 0
    n = start + T - lo
    q, k, v = (torch.randn(a, H, b, device="cuda").to(BF16) for a, b in ((T, dp), (n, dp), (n, vp)))
    gate, scale = torch.randn(T, H, device="cuda").to(BF16), 1.5 / math.sqrt(dp)
    pos = start + torch.arange(T, device="cuda")
    s = torch.einsum("thd,nhd->htn", q.float(), k.float()) * scale
    d = pos[:, None] - (lo + torch.arange(n, device="cuda"))[None]
    s = s.masked_fill(((d < 0) | ((d >= window) if window else d < 0))[None], float("-inf"))
    for sink in (torch.randn(H, device="cuda") * 2, None):
        full = s if sink is None else torch.cat([s, sink[:, None, None].expand(-1, T, 1)], -1)
        want = torch.einsum("htn,nhd->thd", torch.softmax(full, -1)[..., :n], v.float()) * torch.sigmoid(gate.float())[..., None]
        assert rel(_prefill(F, q, k, v, start, lo, window, scale, sink, gate), want) < 5e-3


@pytest.mark.parametrize("window,start", [(64, 0), (128, 300), (200, 57)])
def test_prefill_attention_window_edge(F, window, start):
    """One key with all the weight, at several places of a tile: seen up to window - 1 tokens on and no further."""
    T, H, dp, vp = 400, 1, 64, 64
    lo = max(0, start - window + 1)
    n = start + T - lo
    for key in (start, start + 1, start + 63, start + 127, start + 128, start + 150):
        q, k, v = (torch.randn(a, H, 64, device="cuda") * 0.1 for a in (T, n, n))
        q[..., 0], k[..., 0] = 40.0, 0.0
        k[key - lo, 0, 0], v[..., 1], v[key - lo, 0, 1] = 1.0, 0.0, 5.0
        out = _prefill(F, q.to(BF16), k.to(BF16), v.to(BF16), start, lo, window, 1.0, torch.zeros(H, device="cuda"),
                       torch.full((T, H), 30.0, device="cuda").to(BF16))[:, 0, 1].float()
        seen = torch.arange(start, start + T, device="cuda")
        inside = (seen >= key) & (seen < key + window)
        assert (out[inside] - 5.0).abs().max() < 0.05 and (~inside).any() and out[~inside].abs().max() < 0.1


# ------------------------------------------------------------------------------------------------ model against the oracle
def _want(cfg, w, toks, quant="bf16"):
    return oracle.forward(cfg, kc.quantised(w) if quant == "w8a16" else w, toks)[0]


@pytest.mark.parametrize("quant", ["bf16", "fp32", "w8a16"])
@pytest.mark.parametrize("name", sorted(kc.CASES))
def test_whole_prompt_and_decoding(tmp_path, name, quant):
    """A whole prompt in one step, the same tokens one by one, and a long prompt followed by decoding."""
    folder, cfg, w = kc.model(tmp_path, name)
    n = 150 if name == "one" else 210
    t = kc.tokens(cfg, n)
    want = _want(cfg, w, t, quant)
    eng = kc.engine(folder, quant, "cuda")
    for schedule in ([[("a", n)]], kc.cut("a", n, [1]), kc.cut("a", n, [n - 20] + [1] * 20)):
        got = kc.replay(eng, schedule, {"a": t})["a"]
        assert kc.rms_error(got, want) < TOL[quant], (len(schedule), quant)
    assert eng.model_runner.model.peer_status() == 0


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
@pytest.mark.parametrize("sizes", [[2], [31], [32], [33, 2, 7], [64, 1], [100, 16, 3]])
def test_portions(tmp_path, quant, sizes):
    folder, cfg, w = kc.model(tmp_path, "mixed")
    t = kc.tokens(cfg, 237, seed=2)
    got = kc.replay(kc.engine(folder, quant, "cuda"), kc.cut("a", 237, sizes), {"a": t})["a"]
    assert kc.rms_error(got, _want(cfg, w, t)) < TOL[quant]


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_batches_equal_each_request_alone(tmp_path, name, quant):
    """Portions and single tokens of four requests in one step, pages and slots used again; each request gives what it
    gives alone."""
    folder, cfg, w = kc.model(tmp_path, name)
    p = {r: kc.tokens(cfg, n, seed=n) for r, n in (("a", 150), ("b", 75), ("c", 9), ("d", 130), ("e", 41), ("f", 160))}
    schedule = [[("c", 3), ("a", 100), ("b", 2)], [("b", 1), ("c", 1), ("a", 1)], [("a", 40), ("c", 5), ("b", 33)],
                [("b", 38), ("a", 9)], [("b", 1)], [("d", 64), ("e", 40), ("f", 17)],
                [("d", 1), ("e", 1), ("f", 1)], [("f", 141), ("d", 65)], [("f", 1)]]
    eng = kc.engine(folder, quant, "cuda", blocks=26)
    got = kc.replay(eng, schedule, p)
    for r, t in p.items():
        want = _want(cfg, w, t)
        assert kc.rms_error(got[r], want) < TOL[quant], r
        alone = kc.replay(kc.engine(folder, quant, "cuda", blocks=26, enforce_eager=True), [[(r, len(t))]], {r: t})[r]
        assert kc.rms_error(got[r], alone) < TOL[quant], r
    assert eng.scheduler.block_manager.num_free_blocks == 26


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
def test_influence_ends_with_the_window(tmp_path, quant):
    """One layer with nearly even attention: a changed token changes the logits of exactly the positions whose window
    holds it, in prompts and in decoding, wherever the page borders lie."""
    folder, cfg, w = kc.model(tmp_path, kc.config([kc.layer(2, 32, 24, 40, 35, scale=0.03, ff=64)], width=96, vocab=270))
    t = kc.tokens(cfg, 140)
    eng = kc.engine(folder, quant, "cuda")
    for schedule in ([[("a", 140)]], kc.cut("a", 140, [1]), kc.cut("a", 140, [13])):
        base = kc.replay(eng, schedule, {"a": t})["a"]
        for j in (0, 15, 16, 60):
            u = list(t)
            u[j] = (u[j] + 1) % cfg["vocab"]
            diff = (kc.replay(eng, schedule, {"a": u})["a"] - base).abs().amax(-1)
            assert torch.equal(torch.nonzero(diff > 0).flatten(), torch.arange(j, min(140, j + 35))), j


def test_shared_latents_reach_past_their_owner(tmp_path):
    """A layer that reads another layer's latents has its own, larger window: what it sees is not what the owner sees."""
    cfg = kc.config([kc.layer(2, 32, 24, 40, 3), kc.layer(2, 32, 24, 40, 90, scale=0.9, kv_from=0)], width=96, vocab=270)
    folder, cfg, w = kc.model(tmp_path, cfg)
    t = kc.tokens(cfg, 120)
    want = _want(cfg, w, t)
    for quant in ("bf16", "fp32"):
        for sizes in ([120], [1], [40, 2]):
            got = kc.replay(kc.engine(folder, quant, "cuda"), kc.cut("a", 120, sizes), {"a": t})["a"]
            assert kc.rms_error(got, want) < TOL[quant]


def test_long_decoding_over_many_windows(tmp_path):
    folder, cfg, w = kc.model(tmp_path, "mixed")
    t = kc.tokens(cfg, 640, seed=9)
    want = _want(cfg, w, t)
    got = kc.replay(kc.engine(folder, "fp32", "cuda"), kc.cut("a", 640, [2] + [1] * 638), {"a": t})["a"]
    assert kc.rms_error(got, want) < TOL["fp32"]
    got = kc.replay(kc.engine(folder, "bf16", "cuda"), kc.cut("a", 640, [300] + [1] * 340), {"a": t})["a"]
    assert kc.rms_error(got, want) < TOL["bf16"]


# ------------------------------------------------------------------------------------------------ engine
def _near_greedy(cfg, w, prompt, out, slack):
    full = list(prompt) + list(out)
    lg = _want(cfg, w, full)[len(prompt) - 1:-1]
    return all(float(row.max() - row[t]) <= slack for row, t in zip(lg, out))


@pytest.mark.parametrize("quant,kw", [("fp32", {}), ("bf16", {}), ("bf16", {"max_prefill_chunk_tokens": 32, "num_scheduler_steps": 4}),
                                      ("bf16", {"enforce_eager": True}), ("fp32", {"blocks": 16, "swap_space_bytes": 1 << 24}),
                                      ("fp32", {"blocks": 16})])
def test_generation(tmp_path, quant, kw):
    """Greedy generation through the scheduler: the oracle's tokens in 32-bit, its (nearly) best ones in bf16; with few
    blocks the requests are swapped out or recomputed on the way."""
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = kc.model(tmp_path, "mixed")
    eng = kc.engine(folder, quant, "cuda", **{"blocks": 64, **kw})
    prompts = [kc.tokens(cfg, n, seed=n) for n in (30, 90, 61, 7)]
    outs = eng.generate_token_ids(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert len(o) == 24 and _near_greedy(cfg, w, p, o, 1e-3 if quant == "fp32" else 0.15)
    if kw.get("blocks") == 16:
        assert eng.scheduler.num_preemptions > 0
    eng.close()


def test_sampling_penalties_and_prefix_reuse(tmp_path):
    """Sampled rows with a repetition penalty run on the device path; a cached prefix gives the same greedy tokens."""
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = kc.model(tmp_path, "one")
    eng = kc.engine(folder, "bf16", "cuda", enable_prefix_caching=True)
    prompt = kc.tokens(cfg, 70)
    sp = SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    first = eng.generate_token_ids([prompt], sp)
    assert eng.generate_token_ids([prompt], sp) == first and eng.scheduler.prefix_cache.hit_tokens == 64
    out = eng.generate_token_ids([prompt], SamplingParams(temperature=0.8, top_k=20, repetition_penalty=1.3, max_tokens=8, ignore_eos=True))
    assert len(out[0]) == 8 and all(0 <= t < cfg["vocab"] for t in out[0])


def test_preset_with_default_settings():
    """The preset through the public API in the default (int8) mode."""
    from tileinfer_b200.engine.llm import LLM
    from tileinfer_b200.engine.sampling_params import SamplingParams
    llm = LLM("preset:tiny-kabadra", num_kvcache_blocks=64, max_num_seqs=3, max_model_len=512)
    outs = llm.generate_token_ids([list(range(1, 60)), [5, 6, 7]], SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
    assert [len(o) for o in outs] == [6, 6] and llm.model_runner.model.launches_per_decode_step > 0
    llm.close()


@pytest.mark.parametrize("dtype,tol", [("bfloat16", TOL["bf16"]), ("float32", TOL["fp32"])])
def test_trace_run(tmp_path, dtype, tol):
    cfg = kc.config([kc.layer(2, 16, 16, 24, 9, ff=32), kc.layer(3, 32, 8, 72, 40, ff=32)], width=64, vocab=97)
    folder, cfg, w = kc.model(tmp_path, cfg)
    t, u = kc.tokens(cfg, 60), kc.tokens(cfg, 20, seed=1)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": t[:50], "want": [49]}, {"id": "y", "tokens": u[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": u[3:], "want": [16]}, {"id": "x", "tokens": t[50:51], "want": [0]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": t[51:], "want": [8]}], "end": ["x"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens",
                        "128"], input="\n".join(map(json.dumps, lines)) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = torch.from_numpy(np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4") for i in range(3)]).reshape(4, -1))
    a, b = _want(cfg, w, t), _want(cfg, w, u)
    assert kc.rms_error(got, torch.stack([a[49], b[19], a[50], a[59]])) < tol
