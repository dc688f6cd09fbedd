"""Nogidra on the GPU: each kernel against plain PyTorch fp32, the model against the plain oracle in every precision, and
the engine (portions, batches, reused pages and state slots, long decoding, generation)."""
import json
import math
import os
import subprocess

import numpy as np
import pytest
import torch

import nogidra_cases as nc
import nogidra_oracle as oracle
from test_gerivik_gpu import _paged_kv, _rows, pad64, rel

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = torch.bfloat16, torch.float32


@pytest.fixture(scope="module")
def F():
    from tileinfer_b200.ops import functional
    functional.L("base", "rows", "attention", "latent", "conv", "ssd", "moe")
    return functional


# ------------------------------------------------------------------------------------------------ windowed attention
def _window_ref(q, k, v, pos, scale, window, slopes=None):
    T, H, _ = q.shape
    G = k.shape[1]
    s = torch.einsum("tgad,jgd->gatj", q.float().view(T, G, H // G, -1), k.float()) * scale
    dist = pos.long()[:, None] - torch.arange(k.shape[0], device="cuda")[None]
    if slopes is not None:
        s = s - slopes.view(G, H // G, 1, 1) * dist
    hidden = (dist < 0) | (dist >= window) if window else dist < 0
    a = torch.softmax(s.masked_fill(hidden, float("-inf")), -1)
    return torch.einsum("gatj,jgv->tgav", a, v.float()).reshape(T, H, -1)


def _run_paged(F, q, kc, vc, table, pos, scale, window, slopes=None, gate=None, factor=1.0, nsplit=1, pitch=0, general=False):
    T, H, dp = q.shape
    G, vp = kc.shape[1], vc.shape[2]
    idx, one, zero = (t.int().cuda() for t in (torch.arange(T), torch.ones(T), torch.zeros(T)))
    out = torch.zeros(T, H * vp + pitch, dtype=q.dtype, device="cuda")
    a = F.AttnGeneralParams() if general else F.AttnParams()
    if general:
        a.H, a.G, a.dp, a.vp, a.scale = H, G, dp, vp, scale
    else:
        n = H // G
        a.rep = n // max(d for d in range(1, 17) if n % d == 0)
        a.hq, a.hkv, a.nsplit, a.scale_log2e = H, G, nsplit, scale * math.log2(math.e)
        o = torch.empty(T * G * a.rep * nsplit * 16 * vp, device="cuda")
        ml = torch.empty(T * G * a.rep * nsplit * 32, device="cuda")
        a.o_part, a.ml_part = o.data_ptr(), ml.data_ptr()
    a.q, a.kcache, a.vcache, a.out = q.data_ptr(), kc.data_ptr(), vc.data_ptr(), out.data_ptr()
    a.block_tables, a.positions = table.data_ptr(), pos.data_ptr()
    a.qg_seq, a.qg_tok0, a.qg_ntok = zero.data_ptr(), idx.data_ptr(), one.data_ptr()
    a.max_blocks, a.num_qg, a.num_blocks, a.ldo, a.window, a.out_scale = table.shape[1], T, kc.shape[0], out.stride(0), window, factor
    a.slopes = 0 if slopes is None else slopes.data_ptr()
    if gate is not None:
        a.head_gate, a.ldg, a.gcol = gate.data_ptr(), gate.stride(0), 8
    F.attn_general(a, q.dtype == F32) if general else F.attn_paged(a, dp, vp)
    torch.cuda.synchronize()
    assert not out[:, H * vp:].any()
    return out[:, :H * vp].view(T, H, vp)


def _run_prefill(F, q, kc, vc, table, pos0, scale, window, slopes=None, gate=None, factor=1.0, pitch=0):
    T, H, dp = q.shape
    vp = vc.shape[2]
    pos = (pos0 + torch.arange(T)).int().cuda()
    tiles = torch.tensor([(0, a, min(128, T - a)) for a in range(0, T, 128)], dtype=torch.int32).t().contiguous().cuda()
    out = torch.zeros(T, H * vp + pitch, dtype=BF16, device="cuda")
    F.attn_prefill(q, kc, vc, kc.shape[0], table, pos, tiles, None, out, hq=H, hkv=kc.shape[1], D=dp, DV=vp, max_blocks=table.shape[1], ld=0,
                   scale=scale, window=window, slopes=slopes, head_gate=gate, gcol=8, out_scale=factor)
    torch.cuda.synchronize()
    assert not out[:, H * vp:].any()
    return out[:, :H * vp].view(T, H, vp), pos


# the steepest slopes leave little but the nearest keys: gentle ones keep the far ones in sight
def _slopes(H, kind):
    return None if kind == "flat" else torch.tensor([oracle.slope(h, H) * (1.0 if kind == "steep" else 0.01) for h in range(H)], device="cuda")


@pytest.mark.parametrize("kind", ["flat", "steep", "gentle"])
@pytest.mark.parametrize("H,G,dp,vp,window,nsplit", [(2, 1, 64, 64, 1, 1), (6, 2, 64, 128, 17, 3), (4, 4, 64, 256, 33, 2), (8, 2, 128, 64, 100, 4),
                                                     (34, 2, 128, 256, 250, 1), (40, 2, 256, 64, 0, 2), (3, 3, 256, 128, 300, 7)])
def test_windowed_decode_attention(F, H, G, dp, vp, window, nsplit, kind):
    torch.manual_seed(H + dp)
    n = 411
    q, k, v = (torch.randn(a, b, c, device="cuda").to(BF16) for a, b, c in ((12, H, dp), (n, G, dp), (n, G, vp)))
    pos = torch.tensor([0, 1, 15, 16, 63, 64, 130, 255, 256, 300, 400, 410], dtype=torch.int32, device="cuda")
    kc, vc, table = _paged_kv(k, v, G)
    scale, slopes = 1.5 / math.sqrt(dp), _slopes(H, kind)
    gate = torch.randn(12, 8 + H + 3, device="cuda").to(BF16)
    want = _window_ref(q, k, v, pos, scale, window, slopes) * torch.sigmoid(gate[:, 8:8 + H].float())[..., None] * 0.7
    for general in (False, True):
        got = _run_paged(F, q, kc, vc, table, pos, scale, window, slopes, gate, 0.7, nsplit, 64, general)
        assert rel(got, want) < 6e-3
    q, k, v, gate = (t.float() for t in (q, k, v, gate))
    kc, vc, table = _paged_kv(k, v, G)
    assert rel(_run_paged(F, q, kc, vc, table, pos, scale, window, slopes, gate, 0.7, 1, 64, True), want) < 2e-5


@pytest.mark.parametrize("kind", ["flat", "steep", "gentle"])
@pytest.mark.parametrize("H,G,dp,vp,window,start,T", [(2, 1, 64, 64, 50, 0, 40), (4, 2, 64, 128, 128, 100, 200), (2, 2, 64, 256, 1, 7, 129),
                                                      (4, 1, 128, 64, 129, 300, 333), (4, 2, 128, 128, 16, 0, 300), (1, 1, 128, 256, 300, 64, 130),
                                                      (2, 1, 256, 64, 0, 130, 128), (3, 3, 256, 128, 5, 5, 17), (2, 1, 256, 256, 200, 500, 140)])
def test_windowed_prefill_attention(F, H, G, dp, vp, window, start, T, kind):
    torch.manual_seed(T)
    n = start + T
    q, k, v = (torch.randn(a, b, c, device="cuda").to(BF16) for a, b, c in ((T, H, dp), (n, G, dp), (n, G, vp)))
    kc, vc, table = _paged_kv(k, v, G)
    scale, slopes = 1.5 / math.sqrt(dp), _slopes(H, kind)
    gate = torch.randn(T, 8 + H + 3, device="cuda").to(BF16)
    got, pos = _run_prefill(F, q, kc, vc, table, start, scale, window, slopes, gate, 1.3, 64)
    want = _window_ref(q, k, v, pos, scale, window, slopes) * torch.sigmoid(gate[:, 8:8 + H].float())[..., None] * 1.3
    assert rel(got, want) < 6e-3
    got, _ = _run_prefill(F, q, kc, vc, table, start, scale, window, slopes)
    assert rel(got, _window_ref(q, k, v, pos, scale, window, slopes)) < 6e-3


def test_window_edges_of_one_key_that_stands_out(F):
    """One key carries nearly all the weight: a query sees it while it is window - 1 tokens back and no longer one token on,
    wherever page and tile borders lie, in prompts and in decoding."""
    n = 700
    for key, window in ((0, 17), (15, 128), (16, 129), (127, 200), (128, 1), (300, 333), (431, 16)):
        q, k, v = (torch.randn(n, 1, 64, device="cuda") * 0.1 for _ in range(3))
        q[..., 0], k[..., 0], v[..., 1] = 6.0, 0.0, 0.0
        k[key, 0, 0], v[key, 0, 1] = 6.0, 5.0
        q, k, v = q.to(BF16), k.to(BF16), v.to(BF16)
        kc, vc, table = _paged_kv(k, v, 1, seed=key)
        slopes = torch.full((1,), 1e-4, device="cuda")
        for sl in (None, slopes):
            got, pos = _run_prefill(F, q, kc, vc, table, 0, 0.5, window, sl)
            for o in (got, _run_paged(F, q, kc, vc, table, pos, 0.5, window, sl, nsplit=3), _run_paged(F, q, kc, vc, table, pos, 0.5, window, sl, general=True)):
                seen = o[key:min(n, key + window), 0, 1]
                assert (seen - 5.0).abs().max() < 0.05
                assert o[key + window:].numel() == 0 or o[key + window:, 0, 1].abs().max() < 0.05
                assert key == 0 or o[:key, 0, 1].abs().max() < 0.05


def test_slope_decides_between_two_keys(F):
    """Two equal keys, `d` tokens apart: their weights differ by exp(slope d)."""
    d, slope = 40, torch.tensor([0.05], device="cuda")
    q, k, v = torch.zeros(200, 1, 64, device="cuda"), torch.zeros(200, 1, 64, device="cuda"), torch.zeros(200, 1, 64, device="cuda")
    q[..., 0], k[100, 0, 0], k[100 + d, 0, 0], v[100, 0, 0] = 8.0, 8.0, 8.0, 1.0
    kc, vc, table = _paged_kv(k.to(BF16), v.to(BF16), 1)
    want = 1 / (1 + math.exp(0.05 * d))
    got, pos = _run_prefill(F, q.to(BF16), kc, vc, table, 0, 1.0, 0, slope)
    for o in (got, _run_paged(F, q.to(BF16), kc, vc, table, pos, 1.0, 0, slope, nsplit=2)):
        assert (o[100 + d:, 0, 0] - want).abs().max() < 2e-3 and (o[100:100 + d, 0, 0] - 1).abs().max() < 1e-2


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,G,dim,vdim,dp,vp,rot", [(3, 1, 24, 40, 64, 64, 18), (4, 2, 64, 64, 64, 64, 64), (2, 2, 100, 130, 128, 256, 2),
                                                    (1, 1, 300, 20, 320, 64, 0), (34, 2, 128, 24, 128, 64, 40)])
def test_heads_normed_together_and_store(F, dtype, H, G, dim, vdim, dp, vp, rot):
    torch.manual_seed(dim)
    T, nb, ld = 6, 4, (H + G) * dp + G * vp + 8
    q, k, v = (torch.randn(T, a, b, device="cuda").to(dtype) for a, b in ((H, dim), (G, dim), (G, vdim)))
    qw, kw = torch.rand(H, dim, device="cuda") + 0.5, torch.rand(G, dim, device="cuda") + 0.5
    proj = torch.zeros(T, ld, dtype=dtype, device="cuda")
    proj[:, :(H + G) * dp] = torch.cat([_rows(q, dp), _rows(k, dp)], 1).flatten(1)
    proj[:, (H + G) * dp:(H + G) * dp + G * vp] = _rows(v, vp).flatten(1)
    pos = torch.tensor([0, 1, 17, 1000, 3000, 5], dtype=torch.int32, device="cuda")
    slots = torch.tensor([5, 16, -1, 63, 64, 33], device="cuda")                   # -1 and 64 are not in the cache
    inv = torch.tensor([900.0 ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64).float().cuda()
    qo, kc, vc = torch.zeros(T, H, dp, dtype=dtype, device="cuda"), torch.zeros(nb, G, 16, dp, dtype=dtype, device="cuda"), \
        torch.zeros(nb, G, vp, 16, dtype=dtype, device="cuda")
    qwp, kwp = _rows(qw, dp).flatten().contiguous(), _rows(kw, dp).flatten().contiguous()
    p = F.NormRopeParams()
    p.proj, p.q_w, p.k_w, p.inv_freq, p.positions = proj.data_ptr(), qwp.data_ptr(), kwp.data_ptr(), inv.data_ptr(), pos.data_ptr()
    p.slot_mapping, p.q_out, p.kcache, p.vcache = slots.data_ptr(), qo.data_ptr(), kc.data_ptr(), vc.data_ptr()
    p.T, p.ld, p.q_col, p.k_col, p.v_col, p.H, p.G = T, ld, 0, H * dp, (H + G) * dp, H, G
    p.dim, p.dp, p.vp, p.half, p.num_blocks, p.eps = dim, dp, vp, rot // 2, nb, 1e-4
    F.norm_rope(p, dtype == F32)
    turn = lambda x, w: oracle.rotate_pairs(oracle.unit_rms(x.double().flatten(1), 1e-4).view_as(x).cpu() * w.double().cpu(), pos.cpu(), 900.0, rot).cuda()
    tol = 4e-3 if dtype == BF16 else 2e-4                                           # 32-bit angles of 3000 radians
    assert rel(qo[..., :dim], turn(q, qw)) < tol and not qo[..., dim:].any()
    kwant, vwant = torch.zeros(nb * 16, G, dp, device="cuda"), torch.zeros(nb * 16, G, vp, device="cuda")
    for t in (0, 1, 3, 5):
        kwant[slots[t], :, :dim], vwant[slots[t], :, :vdim] = turn(k, kw)[t].float(), v[t].float()
    assert rel(kc.permute(0, 2, 1, 3).reshape(nb * 16, G, dp), kwant) < tol
    assert torch.equal(vc.permute(0, 3, 1, 2).reshape(nb * 16, G, vp).float(), vwant)


# ------------------------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,R,P,window,nsplit", [(3, 56, 10, 50, 2), (16, 192, 64, 129, 1), (17, 200, 180, 64, 3), (18, 512, 64, 300, 4), (40, 448, 64, 0, 2),
                                                 (5, 512, 64, 1, 1), (2, 513, 30, 70, 1), (33, 500, 70, 200, 3)])
def test_rows_with_a_key_only_part(F, dtype, H, R, P, window, nsplit):
    """The trailing columns of a cache row take part in the scores and not in the output."""
    torch.manual_seed(R + H)
    n, Rp, Ro = 411, pad64(R + P), pad64(R)
    c = _rows(torch.randn(n, R + P, device="cuda"), Rp).to(dtype)
    kc, _, table = _paged_kv(c[:, None], c[:, None], 1)
    pos = torch.tensor([0, 1, 15, 16, 63, 64, 130, 255, 256, 400, 410], dtype=torch.int32, device="cuda")
    T, rows = len(pos), 32 if H > 16 else 16
    q = _rows(torch.randn(T, H, R + P, device="cuda"), Rp).to(dtype)
    split = nsplit if F.latent_attn_splits(Rp, Ro) and dtype == BF16 else 1
    part, ml = torch.empty(T * -(-H // rows) * split * rows * Rp, device="cuda"), torch.empty(T * -(-H // rows) * split * rows * 2, device="cuda")
    idx, one, zero = (t.int().cuda() for t in (torch.arange(T), torch.ones(T), torch.zeros(T)))
    out = torch.full((T, H, Ro), 9.0, dtype=dtype, device="cuda")
    p = F.LatentAttnParams()
    p.q, p.cache, p.out, p.block_tables, p.positions = q.data_ptr(), kc.data_ptr(), out.data_ptr(), table.data_ptr(), pos.data_ptr()
    p.qg_seq, p.qg_tok0, p.qg_ntok, p.o_part, p.ml_part = zero.data_ptr(), idx.data_ptr(), one.data_ptr(), part.data_ptr(), ml.data_ptr()
    p.H, p.R, p.Rp, p.Ro, p.max_blocks, p.nsplit, p.num_qg = H, R, Rp, Ro, table.shape[1], split, T
    p.window, p.num_blocks, p.scale = window, kc.shape[0], 2.0 / math.sqrt(R)
    F.latent_attn(p, dtype == F32)
    torch.cuda.synchronize()
    want = _window_ref(q, c[:, None], c[:, None, :Ro], pos, 2.0 / math.sqrt(R), window)
    assert rel(out, want) < (2e-5 if dtype == F32 else 6e-3)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,dim,rot,R", [(3, 24, 10, 56), (2, 64, 0, 64), (5, 40, 24, 130), (1, 16, 48, 512)])
def test_latents_beside_a_rotated_part(F, dtype, H, dim, rot, R):
    torch.manual_seed(R)
    T, nb, dp, Rp = 6, 4, pad64(dim + rot), pad64(R + rot)
    q, lat, kr = torch.randn(T, H, dim + rot, device="cuda").to(dtype), torch.randn(T, R, device="cuda").to(dtype), torch.randn(T, rot, device="cuda").to(dtype)
    proj = torch.cat([_rows(q, dp).flatten(1), lat, kr, torch.zeros(T, -(R + rot) % 64, dtype=dtype, device="cuda")], 1).contiguous()
    pos = torch.tensor([0, 1, 17, 1000, 3000, 5], dtype=torch.int32, device="cuda")
    slots = torch.tensor([5, 16, -1, 63, 64, 33], device="cuda")
    inv = torch.tensor([900.0 ** (-2 * i / rot) for i in range(rot // 2)], dtype=torch.float64).float().cuda()
    w = torch.rand(R, device="cuda") + 0.5
    cache = torch.full((nb, 16, Rp), 7.0, dtype=dtype, device="cuda")
    F.latent_rope(proj, H, dp, dim, H * dp, w, inv, pos, slots, cache, R, 1e-4)
    turn = lambda x: oracle.rotate_halves(x.double().cpu(), pos.cpu(), 900.0, rot).cuda()
    tol = 4e-3 if dtype == BF16 else 2e-4
    got = proj[:, :H * dp].view(T, H, dp)
    assert torch.equal(got[..., :dim], q[..., :dim]) and not got[..., dim + rot:].any()
    assert rot == 0 or rel(got[..., dim:dim + rot], turn(q[..., dim:])) < tol
    want = torch.full((nb * 16, Rp), 7.0, device="cuda")
    for t in (0, 1, 3, 5):
        want[slots[t]] = 0
        want[slots[t], :R] = (oracle.unit_rms(lat[t].float(), 1e-4) * w)
        want[slots[t], R:R + rot] = turn(kr[:, None])[t, 0].float()
    assert rel(cache.view(-1, Rp), want) < tol


# ------------------------------------------------------------------------------------------------ convolutions
def _conv_setup(dtype, C, taps, lens, seed=0):
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dtype).cuda()
    T, S = sum(lens), len(lens)
    proj = rnd(T, C + 24)
    state = rnd(S + 2, taps - 1, C)
    cu = [sum(lens[:i]) for i in range(S + 1)]
    slots = torch.tensor([S - s for s in range(S)], dtype=torch.int32).cuda()
    return proj, state, cu, slots, rnd(C, taps).float(), rnd(C).float()


def _conv_ref(u, past, w, bias):
    """One sequence: inputs u [n, C] after `past` [taps - 1, C]."""
    return oracle.causal_conv(torch.cat([past, u]).float(), w, bias)[past.shape[0]:]


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
def test_convolution(F, dtype, taps):
    """Portions of many lengths, the inputs carried on, snapshots; then single tokens."""
    for lens in ([1, 2, 3, 40, 17], [1, 1, 1]):
        C, S = 72, len(lens)
        proj, state, cu, slots, w, bias = _conv_setup(dtype, C, taps, lens)
        before, T = state.clone(), sum(lens)
        out = torch.zeros(T, C + 8, dtype=dtype, device="cuda")
        wt = w.t().contiguous()
        p = F.ConvParams()
        p.proj, p.w, p.bias, p.state, p.slots, p.out = proj.data_ptr(), wt.data_ptr(), bias.data_ptr(), state.data_ptr(), slots.data_ptr(), out.data_ptr()
        p.T, p.S, p.ld, p.col, p.C, p.taps, p.ldo, p.silu = T, S, C + 24, 16, C, taps, C + 8, 1
        rel_, idx, snap = torch.zeros(S, 2, dtype=torch.int32), torch.zeros(S, 2, dtype=torch.int32), torch.zeros(3, taps - 1, C, dtype=dtype, device="cuda")
        if max(lens) > 1:
            cut, tiles = torch.tensor(cu, dtype=torch.int32).cuda(), F.conv_tiles(cu).cuda()
            p.cu, p.tiles, p.num_tiles = cut.data_ptr(), tiles.data_ptr(), tiles.shape[1]
            rel_[3], idx[3], rel_[4, 0], idx[4, 0] = torch.tensor([16, 40]), torch.tensor([0, 2]), 1, 1
            rel_, idx = rel_.cuda(), idx.cuda()
            p.snap_rel, p.snap_idx, p.snap, p.num_snap = rel_.data_ptr(), idx.data_ptr(), snap.data_ptr(), 2
        F.conv(p, dtype == F32)
        torch.cuda.synchronize()
        assert not out[:, C:].any()
        for s in range(S):
            u, past = proj[cu[s]:cu[s + 1], 16:16 + C], before[slots[s]]
            want = torch.nn.functional.silu(_conv_ref(u, past, w, bias))
            assert rel(out[cu[s]:cu[s + 1], :C], want) < (4e-3 if dtype == BF16 else 1e-6)
            whole = torch.cat([past, u])
            if taps > 1:
                assert torch.equal(state[slots[s]], whole[len(whole) - taps + 1:])
                for e, (sq, r) in enumerate(((3, 16), (4, 1), (3, 40))):
                    if max(lens) > 1 and sq == s:
                        assert torch.equal(snap[e], whole[r:r + taps - 1])
        rest = [i for i in range(S + 2) if i not in slots.tolist()]
        assert torch.equal(state[rest], before[rest])


@pytest.mark.parametrize("dtype", [BF16, F32])
def test_convolved_heads_and_query_temperature(F, dtype):
    H, G, dp, vp, taps, nb = 3, 1, 64, 128, 3, 5
    C, lens = (H + G) * dp + G * vp, [20, 1, 3]
    proj, state, cu, slots, w, _ = _conv_setup(dtype, C, taps, lens, seed=2)
    before, T = state.clone(), sum(lens)
    pos = torch.cat([torch.arange(5, 25), torch.tensor([0]), torch.arange(60, 63)]).int().cuda()
    slot_map = torch.randperm(nb * 16, generator=torch.Generator().manual_seed(1))[:T].cuda()
    slot_map[4] = -1
    q = torch.zeros(T, H * dp, dtype=dtype, device="cuda")
    kc, vc = torch.zeros(nb, G, 16, dp, dtype=dtype, device="cuda"), torch.zeros(nb, G, vp, 16, dtype=dtype, device="cuda")
    wt, cut, tiles = w.t().contiguous(), torch.tensor(cu, dtype=torch.int32).cuda(), F.conv_tiles(cu).cuda()
    p = F.ConvParams()
    p.proj, p.w, p.state, p.slots, p.cu, p.tiles, p.num_tiles = proj.data_ptr(), wt.data_ptr(), state.data_ptr(), slots.data_ptr(), cut.data_ptr(), tiles.data_ptr(), tiles.shape[1]
    p.positions, p.slot_mapping, p.q_out, p.kcache, p.vcache = pos.data_ptr(), slot_map.data_ptr(), q.data_ptr(), kc.data_ptr(), vc.data_ptr()
    p.T, p.S, p.ld, p.col, p.C, p.taps, p.H, p.G, p.dp, p.vp, p.num_blocks = T, 3, C + 24, 16, C, taps, H, G, dp, vp, nb
    p.temp_coef, p.temp_every = 0.7, 6
    F.conv(p, dtype == F32)
    torch.cuda.synchronize()
    y = torch.cat([_conv_ref(proj[cu[s]:cu[s + 1], 16:16 + C], before[slots[s]], w, None) for s in range(3)])
    temp = torch.tensor([oracle.query_temperature(int(x), 0.7, 6) for x in pos], device="cuda")
    tol = 4e-3 if dtype == BF16 else 1e-6
    assert rel(q, y[:, :H * dp] * temp[:, None]) < tol
    kw, vw = torch.zeros(nb * 16, dp, device="cuda"), torch.zeros(nb * 16, vp, device="cuda")
    for t in range(T):
        if t != 4:
            kw[slot_map[t]], vw[slot_map[t]] = y[t, H * dp:(H + G) * dp], y[t, (H + G) * dp:]
    assert rel(kc.view(-1, dp), kw) < tol and rel(vc.permute(0, 1, 3, 2).reshape(-1, vp), vw) < tol


# ------------------------------------------------------------------------------------------------ state-space mixer
class Ssm:
    """Inputs of the state-space kernels for sequences of the given lengths, and what the plain recurrence makes of them."""

    def __init__(self, F, dtype, H, V, N, G, norm_groups, lens, seed=0, decay=0.0):
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        self.F, self.dtype, self.lens, T = F, dtype, lens, sum(lens)
        self.cu = [sum(lens[:i]) for i in range(len(lens) + 1)]
        self.H, self.V, self.N, self.G, self.vp, self.Np = H, V, N, G, pad64(V), next(s for s in F.SSD_STATE_SIZES if s >= N)
        x, B, C, z, dt = (t.to(dtype).float() for t in (rnd(T, H, V), rnd(T, G, N), rnd(T, G, N), rnd(T, H, V), rnd(T, H)))
        self.A, self.D, bias, norm = rnd(H) * 0.5 + decay, rnd(H), rnd(H) * 0.5, torch.rand(H * V, generator=g) + 0.5
        self.slots = torch.tensor([len(lens) - s for s in range(len(lens))], dtype=torch.int32)
        S0 = rnd(len(lens) + 2, H, N, V)
        self.y, self.states, self.snaps = torch.zeros(T, H, V), S0.clone(), {}
        step = torch.nn.functional.softplus(dt + bias, threshold=1e9)
        for s in range(len(lens)):
            a, b = self.cu[s], self.cu[s + 1]
            for h in range(H):
                k = h // (H // G)
                self.y[a:b, h], self.states[self.slots[s], h] = oracle.state_space(
                    x[a:b, h].double(), B[a:b, k].double(), C[a:b, k].double(), step[a:b, h].double(), self.A[h].double(), self.D[h].double(), S0[self.slots[s], h].double())
        gated = (self.y.double() * torch.nn.functional.silu(z.double())).flatten(1)
        self.out = oracle.group_norm(gated, norm.double(), norm_groups, 1e-4).view(T, H, V)
        wide = H * self.vp
        pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1])).flatten(1)
        self.xbc = torch.cat([pad(x, self.vp), pad(B, self.Np), pad(C, self.Np)], 1).to(dtype).cuda()
        self.proj = torch.cat([torch.zeros(T, 8), pad(z, self.vp), dt, torch.zeros(T, -H % 8)], 1).to(dtype).cuda()
        self.keep = [bias.cuda(), -torch.exp(self.A).cuda(), self.D.cuda(), pad(norm.view(1, H, V), self.vp)[0].cuda(),
                     torch.nn.functional.pad(S0, (0, self.vp - V, 0, self.Np - N)).cuda().contiguous(), self.slots.cuda(),
                     torch.tensor(self.cu, dtype=torch.int32).cuda(), torch.zeros(T, wide).cuda(), torch.full((T, wide + 16), 7.0, dtype=dtype).cuda()]
        p = self.p = F.SsdParams()
        p.xbc, p.proj = self.xbc.data_ptr(), self.proj.data_ptr()
        p.dt_bias, p.neg_a, p.D, p.norm, p.state, p.slots, p.cu, p.y, p.out = (t.data_ptr() for t in self.keep)
        p.ldx, p.ld, p.ldo, p.x_col, p.b_col, p.c_col, p.z_col, p.dt_col = self.xbc.shape[1], self.proj.shape[1], wide + 16, 0, wide, wide + G * self.Np, 8, 8 + wide
        p.H, p.G, p.V, p.vp, p.norm_groups, p.eps = H, G, V, self.vp, norm_groups, 1e-4

    def step(self, seqs=None):
        n = len(self.lens)
        if seqs is not None:
            self._seqs, n = torch.tensor(seqs, dtype=torch.int32).cuda(), len(seqs)
            self.p.seqs = self._seqs.data_ptr()
        self.F.ssd_step(self.p, n, self.Np, self.dtype == F32)

    def chunked(self, seqs, points=None):
        ck, rng = self.F.gla_chunk_table(self.cu, seqs, self.F.ssd_chunk_size(self.Np), points)
        self._ck, self._rng, self._long = ck.cuda(), rng.cuda(), torch.tensor(seqs, dtype=torch.int32).cuda()
        p = self.p
        p.ck_seq, p.ck_tok0, p.ck_ntok, p.ck_snap = (r.data_ptr() for r in self._ck)
        p.long_seq, p.long_ck, p.nc, p.num_long = self._long.data_ptr(), self._rng.data_ptr(), ck.shape[1], len(seqs)
        self._ws = self.F.SsdWorkspace("cuda")
        p.g_ws, p.s_ws = (w.data_ptr() for w in self._ws.get(p.nc, self.H, self.Np, self.vp))
        self.F.ssd_chunked(p, self.Np)

    def check(self, tol, out_tol):
        self.F.ssd_finish(self.p, sum(self.lens), self.dtype == F32)
        torch.cuda.synchronize()
        T, state, y, out = sum(self.lens), self.keep[4], self.keep[7], self.keep[8]
        assert rel(y.view(T, self.H, self.vp)[..., :self.V], self.y.cuda()) < tol
        assert rel(state[..., :self.N, :self.V], self.states.cuda()) < tol and not state[..., self.V:].any() and not state[..., self.N:, :].any()
        got = out[:, :self.H * self.vp].view(T, self.H, self.vp)
        assert rel(got[..., :self.V], self.out.cuda()) < out_tol and not got[..., self.V:].any() and (out[:, self.H * self.vp:] == 7).all()


SSM_SIZES = [(4, 20, 24, 2, 8), (2, 64, 64, 1, 1), (3, 130, 130, 3, 13), (8, 64, 128, 2, 4), (1, 24, 200, 1, 3)]


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,V,N,G,ng", SSM_SIZES + [(2, 40, 300, 2, 2)])
def test_state_space_token_by_token(F, dtype, H, V, N, G, ng):
    x = Ssm(F, dtype, H, V, N, G, ng, [1, 5, 33, 2])
    x.step()
    x.check(1e-5, 4e-3 if dtype == BF16 else 1e-5)
    one = Ssm(F, dtype, H, V, N, G, ng, [1, 1, 1], seed=1)
    one.p.cu = 0                                             # the decode form
    one.step()
    one.check(1e-5, 4e-3 if dtype == BF16 else 1e-5)


# weak decay (states of hundreds of tokens), the usual, and strong (the state is gone within a token)
@pytest.mark.parametrize("decay", [-5.0, 0.0, 3.0])
@pytest.mark.parametrize("H,V,N,G,ng", SSM_SIZES)
def test_state_space_in_chunks(F, H, V, N, G, ng, decay):
    x = Ssm(F, BF16, H, V, N, G, ng, [64, 3, 200, 65, 1, 63], decay=decay)
    x.chunked([0, 2, 3, 5])
    x.step([1, 4])
    x.check(3e-4, 4e-3)


def test_state_space_snapshots(F):
    """States after chosen tokens, from the chunked and the token-serial form."""
    H, V, N = 2, 24, 40
    for chunked in (True, False):
        x = Ssm(F, BF16, H, V, N, 1, 1, [150, 40], seed=4)
        snap = torch.zeros(3, H, 64, 64, device="cuda")
        points = [{48: 0, 128: 2}, {32: 1}]
        rel_, idx = torch.tensor([[48, 128], [32, 0]], dtype=torch.int32).cuda(), torch.tensor([[0, 2], [1, 0]], dtype=torch.int32).cuda()
        x.p.snap_rel, x.p.snap_idx, x.p.snap, x.p.num_snap = rel_.data_ptr(), idx.data_ptr(), snap.data_ptr(), 2
        x.chunked([0, 1], points) if chunked else x.step()
        torch.cuda.synchronize()
        for e, lens in ((0, [48, 40]), (2, [128, 40]), (1, [150, 32])):
            y = Ssm(F, BF16, H, V, N, 1, 1, [150, 40], seed=4)
            s = int(e == 1)
            b = torch.nn.functional.softplus(y.proj[:, y.p.dt_col:y.p.dt_col + H].float() + y.keep[0], threshold=1e9)
            S0 = Ssm(F, BF16, H, V, N, 1, 1, [150, 40], seed=4).keep[4][y.slots[s], :, :N, :V]
            a = y.cu[s]
            for h in range(H):
                B, C = y.xbc[a:a + lens[s], H * 64:H * 64 + N].double(), y.xbc[a:a + lens[s], H * 64 + 64:H * 64 + 64 + N].double()
                want = oracle.state_space(y.xbc[a:a + lens[s], h * 64:h * 64 + V].double(), B, C, b[a:a + lens[s], h].double(), y.A[h].double().cuda(),
                                          y.D[h].double().cuda(), S0[h].double())[1]
                assert rel(snap[e, h, :N, :V], want) < 3e-4


# ------------------------------------------------------------------------------------------------ experts, epilogues
@pytest.mark.parametrize("T,E,top", [(5, 7, 2), (40, 16, 16), (300, 70, 9), (3, 3, 1)])
def test_weights_over_the_chosen_experts(F, T, E, top):
    logits = torch.randn(T, -(-E // 8) * 8, device="cuda") * 3
    g = F.TokenGroups(T, E, E, top, F.moe_counters(E, "cuda"), False, "cuda")
    F.moe_route(g, logits, None, 1, 1)
    z, ids = logits[:, :E].topk(top, -1)
    assert torch.equal(g.ids.view(T, top).sort(-1)[0].long(), ids.sort(-1)[0])
    got = torch.zeros(T, E, device="cuda").scatter_(1, g.ids.view(T, top).long(), g.weight.view(T, top))
    assert rel(got, torch.zeros(T, E, device="cuda").scatter_(1, ids, torch.softmax(z, -1))) < 1e-6


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T", [3, 150])
def test_residual_without_an_output_norm(F, dtype, T):
    W, P = 136, 192
    y, x = _rows(torch.randn(T, W, device="cuda"), P).to(dtype), _rows(torch.randn(T, W, device="cuda"), P)
    w, h = _rows(torch.rand(W, device="cuda") + 0.5, P), torch.zeros(T, P, dtype=dtype, device="cuda")
    for add in (y, None):
        want = x[:, :W] + (0 if add is None else add[:, :W].float())
        F.resid_norm(add, x, None, h, w, W, 1e-4)
        assert rel(x[:, :W], want) < 1e-6
        assert rel(h[:, :W], oracle.unit_rms(want, 1e-4) * w[:W]) < (4e-3 if dtype == BF16 else 1e-6)


@pytest.mark.parametrize("quant", ["bf16", "w8a16", "fp32"])
@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (5, 192, 4160), (130, 328, 192), (700, 4096, 256)])
def test_products_with_biases_and_caps(F, quant, M, N, K):
    from tileinfer_b200.models.products_b200 import Product
    torch.manual_seed(N)
    dt = F32 if quant == "fp32" else BF16
    w, x, b = torch.randn(N, K, device="cuda").to(BF16) / K ** 0.5, torch.randn(M, K, device="cuda").to(dt), torch.randn(N, device="cuda")
    P = Product(w, quant, "cuda")
    dense = w.float() if quant != "w8a16" else P.w.dense().float()
    y = x.float() @ dense.T + b
    tol = 1e-5 if quant == "fp32" else 5e-3
    out = torch.empty(M, N, dtype=dt, device="cuda")
    P(x, out, F.GEPI_STORE, F.gemm_epilogue(bias=b))
    assert rel(out, y) < tol
    act = torch.empty(M, N // 2, dtype=dt, device="cuda")
    P(x, act, F.GEPI_SPLIT_GLU, F.gemm_epilogue(out2=act, n_split=0, glu=(math.inf, 1.0, 0.0), bias=b))
    assert rel(act, torch.nn.functional.silu(y[:, ::2]) * y[:, 1::2]) < tol
    r = torch.randn(M, N, device="cuda")
    want = r + y
    P(x, r, F.GEPI_RESID32, F.gemm_epilogue(resid32=r, bias=b))
    assert rel(r, want) < tol
    lg = torch.empty(M, N, device="cuda")
    P(x, lg, F.GEPI_F32, F.gemm_epilogue(softcap=1.3, scale=2.0))
    assert rel(lg, 1.3 * torch.tanh(2.0 * (y - b) / 1.3)) < tol


# ------------------------------------------------------------------------------------------------ model
def _want(cfg, w, toks):
    return oracle.forward(cfg, w, toks)[0]


@pytest.mark.parametrize("quant", ["fp32", "bf16", "w8a16"])
@pytest.mark.parametrize("name", sorted(nc.CASES))
def test_prompts_and_decoding_match_oracle(tmp_path, name, quant):
    """Whole prompts, and the same tokens one by one, against the plain equations."""
    folder, cfg, w = nc.model(tmp_path, name, decisive=quant != "fp32")
    t = nc.tokens(cfg, 211)
    want = _want(cfg, nc.quantised(w) if quant == "w8a16" else w, t)
    eng = nc.engine(folder, quant, "cuda")
    for sizes in ([211], [150, 1]):
        nc.assert_close(nc.replay(eng, nc.cut("a", 211, sizes), {"a": t})["a"], want, quant)
    nc.assert_close(nc.replay(eng, nc.cut("a", 40, [1]), {"a": t[:40]})["a"], want[:40], quant)
    eng.close()


def test_residual_stream_layer_by_layer(tmp_path):
    """The residual after every layer: the model cut off behind it, with a head that shows the stream."""
    folder, cfg, w = nc.model(tmp_path, "mixed")
    t = nc.tokens(cfg, 60)
    stream = oracle.forward(cfg, w, t)[1]
    from tileinfer_b200.models.checkpoint import CheckpointWeights
    from tileinfer_b200.models.mixed_b200 import B200MixedModel
    from tileinfer_b200.models.nogidra import NogidraConfig
    from tileinfer_b200.models.reference_cpu import Batch
    for n in range(1, len(cfg["layers"]) + 1):
        mc = NogidraConfig.from_dict(dict(cfg, layers=cfg["layers"][:n]))
        m = B200MixedModel(mc, CheckpointWeights(mc, folder), quant="fp32")
        m.alloc_cache(8, 16, 2)
        b = Batch(torch.tensor(t), torch.arange(60), [0, 60], [60], [[5, 2, 7, 0]], torch.tensor([[5, 2, 7, 0][j // 16] * 16 + j % 16 for j in range(60)]),
                  [1], out_rows=list(range(60)))
        assert rel(m.forward(b)[:, :cfg["width"]].cpu(), stream[n - 1]) < 1e-5


def test_free_choice_of_experts_in_16_bit(tmp_path):
    """With routers that decide freely a rounding may move a token to another expert: most positions agree."""
    folder, cfg, w = nc.model(tmp_path, "mixed")
    t = nc.tokens(cfg, 200)
    want = _want(cfg, w, t)
    for sizes in ([200], [50, 1]):
        d = nc.errors(nc.replay(nc.engine(folder, "bf16", "cuda"), nc.cut("a", 200, sizes), {"a": t})["a"], want)
        assert d.quantile(0.5) < 0.03 and d.quantile(0.9) < 0.3


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
@pytest.mark.parametrize("sizes", [[2], [31], [32], [33, 2, 7], [64, 1], [100, 16, 3]])
def test_portions(tmp_path, quant, sizes):
    folder, cfg, w = nc.model(tmp_path, "mixed", decisive=quant == "bf16")
    t = nc.tokens(cfg, 237, seed=2)
    got = nc.replay(nc.engine(folder, quant, "cuda"), nc.cut("a", 237, sizes), {"a": t})["a"]
    nc.assert_close(got, _want(cfg, w, t), quant)


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_batches_equal_each_request_alone(tmp_path, name, quant):
    """Portions and single tokens of four requests in one step, pages and slots used again; each request gives what it
    gives alone."""
    folder, cfg, w = nc.model(tmp_path, name, decisive=quant == "bf16")
    p = {r: nc.tokens(cfg, n, seed=n) for r, n in (("a", 150), ("b", 75), ("c", 9), ("d", 130), ("e", 41), ("f", 160))}
    schedule = [[("c", 3), ("a", 100), ("b", 2)], [("b", 1), ("c", 1), ("a", 1)], [("a", 40), ("c", 5), ("b", 33)],
                [("b", 38), ("a", 9)], [("b", 1)], [("d", 64), ("e", 40), ("f", 17)],
                [("d", 1), ("e", 1), ("f", 1)], [("f", 141), ("d", 65)], [("f", 1)]]
    eng = nc.engine(folder, quant, "cuda", blocks=26)
    got = nc.replay(eng, schedule, p)
    for r, t in p.items():
        nc.assert_close(got[r], _want(cfg, w, t), quant)
        alone = nc.replay(nc.engine(folder, quant, "cuda", blocks=26, enforce_eager=True), [[(r, len(t))]], {r: t})[r]
        nc.assert_close(got[r], alone, quant)
    assert eng.scheduler.block_manager.num_free_blocks == 26 and len(eng.model_runner.free_deltanet_slots) == 4


@pytest.mark.parametrize("layer", [nc.latent(2, 24, 8, 16, 40, 30), nc.latent(2, 24, 8, 16, 512, 130), nc.attention(2, 1, 24, 40, 1, 30),
                                   nc.attention(2, 1, 24, 40, 3, 129), nc.parallel(nc.normed(2, 1, 24, 40, 24, 33), nc.ssm(1, 8, 8, 1, 1, 1), right_scale=0.0)])
def test_what_a_token_reaches(tmp_path, layer):
    """One layer, one changed token: the logits change for exactly as many tokens as the window (and the convolution behind
    it) reaches, in prompts and in decoding, and by as much as the oracle says."""
    cfg = nc.config([layer], width=96, vocab=200)
    folder, cfg, w = nc.model(tmp_path, cfg)
    t, at = nc.tokens(cfg, 180), 21
    u = t[:at] + [(t[at] + 1) % cfg["vocab"]] + t[at + 1:]
    change = _want(cfg, w, u) - _want(cfg, w, t)
    m = layer["mixer"].get("left", layer["mixer"])
    reach = at + m["mask"]["size"] + m.get("conv", 1) - 1
    assert change[at:reach].abs().amax(-1).min() > 1e-6 and not change[reach:].any()
    eng = nc.engine(folder, "fp32", "cuda")
    for sizes in ([180], [60, 1], [13]):
        d = nc.replay(eng, nc.cut("a", 180, sizes), {"a": u})["a"] - nc.replay(eng, nc.cut("a", 180, sizes), {"a": t})["a"]
        assert rel(d, change) < 1e-2 and not d[:at].any() and not d[reach:].any()


def test_slow_states_carry_the_first_token(tmp_path):
    """With hardly any decay a changed first token changes the logits hundreds of tokens later, by as much as the oracle says."""
    cfg = nc.config([nc.parallel(nc.normed(1, 1, 16, 16, 16, 4), nc.ssm(2, 24, 32, 1, 4, 1), left_scale=0.0)], width=96, vocab=200)
    w = oracle.random_weights(cfg, 3)
    w["l0.mix.right.A_log"] = torch.full_like(w["l0.mix.right.A_log"], -7.0)
    folder = oracle.write_model(str(tmp_path / "m"), cfg, w)
    t = nc.tokens(cfg, 400)
    u = [(t[0] + 1) % cfg["vocab"]] + t[1:]
    change = _want(cfg, w, u) - _want(cfg, w, t)
    for quant, tol in (("fp32", 2e-2), ("bf16", 0.5)):
        eng = nc.engine(folder, quant, "cuda")
        for sizes in ([400], [350, 1], [70]):
            d = nc.replay(eng, nc.cut("a", 400, sizes), {"a": u})["a"] - nc.replay(eng, nc.cut("a", 400, sizes), {"a": t})["a"]
            assert change[300:].abs().max() > 1e-2 and rel(d[300:], change[300:]) < tol


def test_long_decoding(tmp_path):
    for quant in ("fp32", "bf16"):
        folder, cfg, w = nc.model(tmp_path / quant, "mixed", decisive=quant == "bf16")
        t = nc.tokens(cfg, 640, seed=9)
        got = nc.replay(nc.engine(folder, quant, "cuda"), nc.cut("a", 640, [2 if quant == "fp32" else 300] + [1] * 638), {"a": t})["a"]
        nc.assert_close(got, _want(cfg, w, t), quant)


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
    blocks the requests are swapped out with their states or recomputed on the way."""
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = nc.model(tmp_path, "mixed", decisive=quant == "bf16")
    eng = nc.engine(folder, quant, "cuda", **{"blocks": 64, **kw})
    prompts = [nc.tokens(cfg, n, seed=n) for n in (30, 90, 61, 7)]
    outs = eng.generate_token_ids(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert len(o) == 24 and _near_greedy(cfg, w, p, o, 1e-3 if quant == "fp32" else 0.2)
    if kw.get("blocks") == 16:
        assert eng.scheduler.num_preemptions > 0
    eng.close()


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
@pytest.mark.parametrize("name", ["one", "latent_only"])
def test_prefix_reuse(tmp_path, name, quant):
    """A cached prefix (pages, and for recurrent models a snapshot of states and convolution inputs) gives the tokens that a
    full prefill gives."""
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = nc.model(tmp_path, name, decisive=quant == "bf16")
    eng = nc.engine(folder, quant, "cuda", enable_prefix_caching=True)
    base, sp = nc.tokens(cfg, 130), SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    eng.generate_token_ids([base], sp)
    for n in (129, 130):
        prompt = base[:n] + nc.tokens(cfg, 21, seed=n)
        out = eng.generate_token_ids([prompt], sp)[0]
        assert _near_greedy(cfg, w, prompt, out, 1e-3 if quant == "fp32" else 0.2)
    assert eng.scheduler.prefix_cache.hit_tokens == 256


def test_sampling_with_penalties(tmp_path):
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = nc.model(tmp_path, "one")
    eng = nc.engine(folder, "bf16", "cuda")
    out = eng.generate_token_ids([nc.tokens(cfg, 70)], SamplingParams(temperature=0.8, top_k=20, repetition_penalty=1.3, max_tokens=8, ignore_eos=True))
    assert len(out[0]) == 8 and all(0 <= t < cfg["vocab"] for t in out[0])


def test_preset_with_default_settings():
    """The preset through the public API in the default (int8) mode."""
    from tileinfer_b200.engine.llm import LLM
    from tileinfer_b200.engine.sampling_params import SamplingParams
    llm = LLM("preset:tiny-nogidra", num_kvcache_blocks=64, max_num_seqs=3, max_model_len=512)
    outs = llm.generate_token_ids([list(range(1, 60)), [5, 6, 7]], SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
    assert [len(o) for o in outs] == [6, 6] and llm.model_runner.model.launches_per_decode_step > 0
    llm.close()


@pytest.mark.parametrize("dtype,quant", [("bfloat16", "bf16"), ("float32", "fp32")])
def test_trace_run(tmp_path, dtype, quant):
    folder, cfg, w = nc.model(tmp_path, "one", decisive=dtype == "bfloat16")
    t, u = nc.tokens(cfg, 60), nc.tokens(cfg, 20, seed=1)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": t[:50], "want": [49]}, {"id": "y", "tokens": u[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": u[3:], "want": [16]}, {"id": "x", "tokens": t[50:51], "want": [0]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": t[51:], "want": [8]}], "end": ["x"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens",
                        "128"], input="\n".join(map(json.dumps, lines)) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = torch.from_numpy(np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4") for i in range(3)]).reshape(4, -1))
    a, b = _want(cfg, w, t), _want(cfg, w, u)
    nc.assert_close(got, torch.stack([a[49], b[19], a[50], a[59]]), quant)
