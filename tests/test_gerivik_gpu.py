"""Gerivik on the GPU: each kernel against plain PyTorch fp32, the model against the plain oracle in every precision, and
the engine (portions, batches, reused pages and state slots, long decoding, generation)."""
import json
import math
import os
import subprocess

import numpy as np
import pytest
import torch

import gerivik_cases as gc
import gerivik_oracle as oracle

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = torch.bfloat16, torch.float32


@pytest.fixture(scope="module")
def F():
    from tileinfer_b200.ops import functional
    functional.L("base", "rows", "attention", "gla", "moe")
    return functional


def rel(got, want):
    return ((got.float() - want.float()).norm() / want.float().norm().clamp_min(1e-20)).item()


def _rows(t, pitch):
    out = torch.zeros(*t.shape[:-1], pitch, dtype=t.dtype, device=t.device)
    out[..., :t.shape[-1]] = t
    return out


def pad64(n):
    return -(-n // 64) * 64


# ------------------------------------------------------------------------------------------------ row operations
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("W", [40, 136, 1500, 2056, 9000])
def test_residual_and_norms(F, dtype, W):
    P, T = pad64(W), 7
    torch.manual_seed(W)
    y = _rows(torch.randn(T, W, device="cuda").to(dtype), P)
    x = _rows(torch.randn(T, W, device="cuda") * 3, P)
    a, b = (_rows(torch.rand(W, device="cuda") + 0.5, P) for _ in range(2))
    want = x[:, :W] + oracle.rms_norm(y[:, :W].float(), a[:W], 1e-3)
    h = torch.full((T, P), 7.0, dtype=dtype, device="cuda")
    F.resid_norm(y, x, a, h, b, W, 1e-3)
    assert rel(x[:, :W], want) < 1e-6 and not x[:, W:].any()
    assert rel(h[:, :W], oracle.rms_norm(want, b[:W], 1e-3)) < (1e-6 if dtype == F32 else 4e-3) and not h[:, W:].any()
    before = h.clone()
    F.resid_norm(y, x, a, h, None, W, 1e-3)                  # the last layer: no next norm
    assert torch.equal(h, before)


def test_scaled_embedding(F):
    e, ids = torch.randn(50, 128, device="cuda").to(BF16), torch.tensor([3, 49, 0], device="cuda")
    x, pos = torch.empty(3, 128, device="cuda"), torch.zeros(3, dtype=torch.int32, device="cuda")
    F.embed_pos(ids, pos, e, None, None, x, 100, 1e-3, scale=12.5)
    assert torch.equal(x, e[ids].float() * 12.5)


# ------------------------------------------------------------------------------------------------ attention kernels
def _paged_kv(k, v, G, seed=0):
    """k [n, G, dp], v [n, G, vp] of one sequence in shuffled pages of a larger cache; everything else holds large values."""
    n, nb = k.shape[0], -(-k.shape[0] // 16)
    table = torch.randperm(nb + 5, generator=torch.Generator().manual_seed(seed))[:nb]
    kc = torch.full((nb + 5, G, 16, k.shape[-1]), 50.0, dtype=k.dtype, device="cuda")
    vc = torch.full((nb + 5, G, v.shape[-1], 16), 50.0, dtype=v.dtype, device="cuda")
    for j in range(n):
        kc[table[j // 16], :, j % 16] = k[j]
        vc[table[j // 16], :, :, j % 16] = v[j]
    return kc, vc, table.int().cuda()[None].contiguous()


def _capped_ref(q, k, v, pos, scale, cap):
    T, H, _ = q.shape
    G = k.shape[1]
    s = torch.einsum("tgad,jgd->gatj", q.float().view(T, G, H // G, -1), k.float()) * scale
    s = cap * torch.tanh(s / cap)
    later = pos[:, None] < torch.arange(k.shape[0], device="cuda")[None]
    a = torch.softmax(s.masked_fill(later, float("-inf")), -1)
    return torch.einsum("gatj,jgv->tgav", a, v.float()).reshape(T, H, -1)


def _run_paged(F, q, kc, vc, table, pos, scale, cap, nsplit, general=False):
    T, H, dp = q.shape
    G, vp = kc.shape[1], vc.shape[2]
    idx, one, zero = (t.int().cuda() for t in (torch.arange(T), torch.ones(T), torch.zeros(T)))
    out = torch.zeros(T, H * vp, dtype=q.dtype, device="cuda")
    if general:
        a = F.AttnGeneralParams()
        a.H, a.G, a.dp, a.vp, a.ldo, a.scale, a.softcap = H, G, dp, vp, H * vp, scale, cap
    else:
        a, n = F.AttnParams(), H // G
        a.rep = n // max(d for d in range(1, 17) if n % d == 0)
        a.hq, a.hkv, a.nsplit = H, G, nsplit
        a.cap_in, a.cap_out = 2 * scale / cap * math.log2(math.e), cap * math.log2(math.e)
        o = torch.empty(T * G * a.rep * nsplit * 16 * vp, device="cuda")
        ml = torch.empty(T * G * a.rep * nsplit * 32, device="cuda")
        a.o_part, a.ml_part = o.data_ptr(), ml.data_ptr()
    a.q, a.kcache, a.vcache, a.out = q.data_ptr(), kc.data_ptr(), vc.data_ptr(), out.data_ptr()
    a.block_tables, a.positions = table.data_ptr(), pos.data_ptr()
    a.qg_seq, a.qg_tok0, a.qg_ntok = zero.data_ptr(), idx.data_ptr(), one.data_ptr()
    a.max_blocks, a.num_qg, a.num_blocks = table.shape[1], T, kc.shape[0]
    F.attn_general(a, q.dtype == F32) if general else F.attn_paged(a, dp, vp)
    torch.cuda.synchronize()
    return out.view(T, H, vp)


@pytest.mark.parametrize("H,G,dp,vp,nsplit", [(2, 1, 64, 64, 1), (6, 2, 64, 128, 3), (4, 4, 64, 256, 2), (8, 2, 128, 64, 4), (16, 4, 128, 128, 5),
                                              (34, 2, 128, 256, 1), (40, 2, 256, 64, 2), (3, 3, 256, 128, 7), (4, 2, 256, 256, 32)])
@pytest.mark.parametrize("cap", [1.5, 30.0])
def test_capped_decode_attention(F, H, G, dp, vp, nsplit, cap):
    torch.manual_seed(H + dp)
    n = 411
    q, k, v = (torch.randn(a, b, c, device="cuda").to(BF16) for a, b, c in ((11, H, dp), (n, G, dp), (n, G, vp)))
    pos = torch.tensor([0, 1, 15, 16, 63, 64, 130, 255, 256, 400, 410], dtype=torch.int32, device="cuda")
    kc, vc, table = _paged_kv(k, v, G)
    scale = 2.5 / math.sqrt(dp)
    want = _capped_ref(q, k, v, pos, scale, cap)
    assert rel(_run_paged(F, q, kc, vc, table, pos, scale, cap, nsplit), want) < 6e-3
    assert rel(_run_paged(F, q, kc, vc, table, pos, scale, cap, 1, general=True), want) < 6e-3


@pytest.mark.parametrize("H,G,dp,vp", [(2, 1, 64, 64), (6, 2, 64, 192), (34, 2, 128, 320), (3, 1, 320, 64), (2, 2, 576, 704)])
def test_plain_attention_in_32_bit(F, H, G, dp, vp):
    torch.manual_seed(dp)
    q, k, v = (torch.randn(a, b, c, device="cuda") for a, b, c in ((7, H, dp), (300, G, dp), (300, G, vp)))
    pos = torch.tensor([0, 15, 16, 100, 255, 256, 299], dtype=torch.int32, device="cuda")
    kc, vc, table = _paged_kv(k, v, G)
    got = _run_paged(F, q, kc, vc, table, pos, 2.5 / math.sqrt(dp), 4.0, 1, general=True)
    assert rel(got, _capped_ref(q, k, v, pos, 2.5 / math.sqrt(dp), 4.0)) < 2e-5


def _run_prefill(F, q, kc, vc, table, pos0, scale, cap, qk_max):
    T, H, dp = q.shape
    pos = (pos0 + torch.arange(T)).int().cuda()
    tiles = torch.tensor([(0, a, min(128, T - a)) for a in range(0, T, 128)], dtype=torch.int32).t().contiguous().cuda()
    out = torch.zeros(T, H * vc.shape[2], dtype=BF16, device="cuda")
    F.attn_prefill(q, kc, vc, kc.shape[0], table, pos, tiles, None, out, hq=H, hkv=kc.shape[1], D=dp, DV=vc.shape[2],
                   max_blocks=table.shape[1], ld=0, scale=scale, softcap=cap, qk_max=qk_max)
    torch.cuda.synchronize()
    return out.view(T, H, -1), pos


# cap 45 with unit heads: bounded scores, the series and no running maximum; cap 1.5: the exact form
@pytest.mark.parametrize("H,G,dp,vp,start,T", [(2, 1, 64, 64, 0, 40), (4, 2, 64, 128, 100, 200), (2, 2, 64, 256, 7, 129), (4, 1, 128, 64, 300, 333),
                                               (4, 2, 128, 128, 0, 300), (1, 1, 128, 256, 64, 130), (2, 1, 256, 64, 0, 128), (3, 3, 256, 128, 5, 17),
                                               (2, 1, 256, 256, 500, 140)])
@pytest.mark.parametrize("cap", [1.5, 45.0])
def test_capped_prefill_attention(F, H, G, dp, vp, start, T, cap):
    torch.manual_seed(T)
    n = start + T
    q, k = (oracle.unit_rms(torch.randn(a, b, dp, device="cuda"), 1e-6).to(BF16) for a, b in ((T, H), (n, G)))
    v = torch.randn(n, G, vp, device="cuda").to(BF16)
    kc, vc, table = _paged_kv(k, v, G)
    scale = dp ** -0.5
    for bound in (0.0, 1.02 * dp):
        got, pos = _run_prefill(F, q, kc, vc, table, start, scale, cap, bound)
        assert rel(got, _capped_ref(q, k, v, pos, scale, cap)) < 6e-3


def test_one_far_key_stands_out(F):
    """One key carries nearly all the weight of every later query, however far back it is and wherever its page and tile
    borders lie; earlier queries do not see it."""
    n, dp = 700, 64
    for key in (0, 15, 16, 127, 128, 400):
        q, k, v = (torch.randn(n, 1, 64, device="cuda") * 0.1 for _ in range(3))
        q[..., 0], k[..., 0], v[..., 1] = 6.0, 0.0, 0.0
        k[key, 0, 0], v[key, 0, 1] = 6.0, 5.0
        q, k, v = q.to(BF16), k.to(BF16), v.to(BF16)
        kc, vc, table = _paged_kv(k, v, 1, seed=key)
        got, pos = _run_prefill(F, q, kc, vc, table, 0, 0.5, 40.0, 0.0)
        assert (got[key:, 0, 1] - 5.0).abs().max() < 0.05 and (key == 0 or got[:key, 0, 1].abs().max() < 0.05)
        got = _run_paged(F, q, kc, vc, table, pos, 0.5, 40.0, 3)
        assert (got[key:, 0, 1] - 5.0).abs().max() < 0.05 and (key == 0 or got[:key, 0, 1].abs().max() < 0.05)


def test_tanh_of_capped_scores(F):
    """Single-key prompts see nothing of a score; two keys reveal their difference: the weight ratio follows the cap."""
    cap, dp = 2.0, 64
    for s in (-3.9, -1.0, 0.3, 0.9, 6.0):                  # |s / cap| on both sides of the series' range
        q, k, v = (torch.zeros(2, 1, dp, device="cuda") for _ in range(3))
        q[1, 0, 0], k[0, 0, 0], v[0, 0, 0] = 1.0, s, 1.0
        kc, vc, table = _paged_kv(k.to(BF16), v.to(BF16), 1)
        want = torch.sigmoid(torch.tensor(cap * math.tanh(float(k.to(BF16)[0, 0, 0]) / cap)))
        for bound in (0.0, abs(s) * 1.01):
            got, pos = _run_prefill(F, q.to(BF16), kc, vc, table, 0, 1.0, cap, bound)
            assert abs(float(got[1, 0, 0]) - float(want)) < 3e-3
        assert abs(float(_run_paged(F, q.to(BF16), kc, vc, table, pos, 1.0, cap, 1)[1, 0, 0]) - float(want)) < 3e-3


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,G,dim,vdim,dp,vp,rot", [(3, 1, 24, 40, 64, 64, 18), (4, 2, 64, 64, 64, 64, 64), (2, 2, 100, 130, 128, 256, 2), (1, 1, 300, 20, 320, 64, 0)])
def test_rotated_unit_heads_and_store(F, dtype, H, G, dim, vdim, dp, vp, rot):
    torch.manual_seed(dim)
    T, nb = 6, 4
    ld = (H + G) * dp + G * vp + 8
    q, k, v = (torch.randn(T, a, b, device="cuda").to(dtype) for a, b in ((H, dim), (G, dim), (G, vdim)))
    proj = torch.zeros(T, ld, dtype=dtype, device="cuda")
    proj[:, :(H + G) * dp] = torch.cat([_rows(q, dp), _rows(k, dp)], 1).flatten(1)
    proj[:, (H + G) * dp:(H + G) * dp + G * vp] = _rows(v, vp).flatten(1)
    pos = torch.tensor([0, 1, 17, 1000, 70000, 5], dtype=torch.int32, device="cuda")
    slots = torch.tensor([5, 16, -1, 63, 64, 33], device="cuda")                   # -1 and 64 are not in the cache
    inv = torch.tensor([900.0 ** (-2 * i / rot) for i in range(rot // 2)] or [0.0], dtype=torch.float64).float().cuda()
    qo, kc, vc = torch.zeros(T, H, dp, dtype=dtype, device="cuda"), torch.zeros(nb, G, 16, dp, dtype=dtype, device="cuda"), \
        torch.zeros(nb, G, vp, 16, dtype=dtype, device="cuda")
    p = F.RopeUnitParams()
    p.proj, p.inv_freq, p.positions, p.slot_mapping = proj.data_ptr(), inv.data_ptr(), pos.data_ptr(), slots.data_ptr()
    p.q_out, p.kcache, p.vcache = qo.data_ptr(), kc.data_ptr(), vc.data_ptr()
    p.T, p.ld, p.q_col, p.k_col, p.v_col, p.H, p.G = T, ld, 0, H * dp, (H + G) * dp, H, G
    p.dim, p.dp, p.vp, p.half, p.num_blocks, p.eps = dim, dp, vp, rot // 2, nb, 1e-4
    F.rope_unit(p, dtype == F32)
    turn = lambda x: oracle.unit_rms(oracle.rotate(x.double().cpu(), pos.cpu(), 900.0, rot), 1e-4).cuda()
    tol = 4e-3 if dtype == BF16 else 3e-3                                           # 32-bit angles: 70000 radians to 4e-3
    near = [0, 1, 2, 3, 5]
    assert rel(qo[near][..., :dim], turn(q)[near]) < (4e-3 if dtype == BF16 else 3e-5) and not qo[..., dim:].any()
    assert rel(qo[..., :dim], turn(q)) < tol
    kw, vw = torch.zeros(nb * 16, G, dp, device="cuda"), torch.zeros(nb * 16, G, vp, device="cuda")
    for t in (0, 1, 3, 5):
        kw[slots[t], :, :dim], vw[slots[t], :, :vdim] = turn(k)[t].float(), v[t].float()
    assert rel(kc.permute(0, 2, 1, 3).reshape(nb * 16, G, dp), kw) < (4e-3 if dtype == BF16 else 3e-5)
    assert torch.equal(vc.permute(0, 3, 1, 2).reshape(nb * 16, G, vp).float(), vw)


# ------------------------------------------------------------------------------------------------ gated linear attention
class Gla:
    """Random inputs of the recurrence kernels in their layout, and the oracle's outputs and states."""

    def __init__(self, F, lens, H, dim, vdim, R, tau, dtype, bias=0.0, seed=0):
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        self.F, self.lens, self.H, self.dim, self.vdim, self.tau, self.dtype = F, lens, H, dim, vdim, tau, dtype
        self.dp, self.vp = next(s for s in F.GLA_KEY_SIZES if s >= dim), pad64(vdim)
        T = self.T = sum(lens)
        self.q, self.k, self.v, self.g = (rnd(T, H, n).to(dtype).float() for n in (dim, dim, vdim, vdim))
        self.a1, self.a2 = rnd(T, R).to(dtype).float(), rnd(H * dim, R) / math.sqrt(R)
        self.bias, self.norm = rnd(H * dim) + bias, torch.rand(vdim, generator=g) + 0.5
        self.alpha = oracle.channel_decay(self.a1, torch.eye(R), self.a2, self.bias, tau).view(T, H, dim)
        self.start = rnd(len(lens) + 2, H, dim, vdim)                               # the states before
        pad = lambda t, n: _rows(t, n).flatten(1)
        cols = [pad(self.q, self.dp), pad(self.k, self.dp), pad(self.v, self.vp), pad(self.g, self.vp), _rows(self.a1, -(-R // 8) * 8)]
        self.proj = torch.cat(cols, 1).to(dtype).cuda().contiguous()
        self.state = torch.zeros(len(lens) + 2, H, self.dp, self.vp)
        self.state[:, :, :dim, :vdim] = self.start
        self.state = self.state.cuda()
        self.slots = torch.randperm(len(lens) + 2, generator=g)[:len(lens)].int().cuda()
        self.cu = torch.tensor([0] + lens).cumsum(0).int().cuda()
        a2 = torch.zeros(H, self.dp, R)
        a2[:, :dim] = self.a2.view(H, dim, R)
        self.dev = [a2.reshape(-1, R).t().contiguous().cuda(), _rows(self.bias.view(H, dim), self.dp).flatten().cuda(), _rows(self.norm[None], self.vp)[0].cuda()]
        self.o = torch.zeros(T, H * self.vp, device="cuda")
        self.out = torch.zeros(T, H * self.vp, dtype=dtype, device="cuda")
        p = self.p = F.GlaParams()
        p.proj, p.a2, p.a2_bias, p.norm, p.state = self.proj.data_ptr(), *(t.data_ptr() for t in self.dev), self.state.data_ptr()
        p.slots, p.cu, p.o, p.out = self.slots.data_ptr(), self.cu.data_ptr(), self.o.data_ptr(), self.out.data_ptr()
        p.ld, p.ldo, p.H, p.R, p.vdim = self.proj.shape[1], self.out.shape[1], H, R, vdim
        p.k_col, p.v_col = H * self.dp, 2 * H * self.dp
        p.g_col, p.a_col = p.v_col + H * self.vp, p.v_col + 2 * H * self.vp
        p.q_scale, p.inv_tau, p.eps = dim ** -0.5, 1.0 / tau, 1e-5

    def chunked(self, points=None):
        F, p = self.F, self.p
        ck, rng = F.gla_chunk_table(self.cu.tolist(), list(range(len(self.lens))), F.gla_chunk_size(self.dp), points)
        self.keep = [ck.cuda(), rng.cuda(), torch.arange(len(self.lens)).int().cuda(), F.GlaWorkspace("cuda")]
        p.ck_seq, p.ck_tok0, p.ck_ntok, p.ck_snap = (r.data_ptr() for r in self.keep[0])
        p.long_ck, p.long_seq, p.nc, p.num_long = self.keep[1].data_ptr(), self.keep[2].data_ptr(), ck.shape[1], len(self.lens)
        p.g_ws, p.s_ws = (t.data_ptr() for t in self.keep[3].get(p.nc, self.H, self.dp, self.vp))
        F.gla_chunked(p, self.dp, self.vp)

    def serial(self):
        self.F.gla_step(self.p, len(self.lens), self.dp, self.vp, self.dtype == F32)

    def want(self):
        """(outputs [T, H, vdim], states by sequence, states after every token) in float64."""
        o, S, every = torch.zeros(self.T, self.H, self.vdim), [], []
        for i, s in enumerate(self.slots.tolist()):
            a, b = int(self.cu[i]), int(self.cu[i + 1])
            states, per = [], []
            for h in range(self.H):
                st, run = self.start[s, h].double(), []
                for t in range(a, b):
                    y, st = oracle.recurrence(self.q[t:t + 1, h].double() * self.dim ** -0.5, self.k[t:t + 1, h].double(), self.v[t:t + 1, h].double(),
                                              self.alpha[t:t + 1, h].double(), st)
                    o[t, h] = y[0]
                    run.append(st)
                states.append(st)
                per.append(torch.stack(run))
            S.append(torch.stack(states))
            every.append(torch.stack(per, 1))
        return o, S, every

    def check(self, tol):
        o, S, every = self.want()
        got = self.o.view(self.T, self.H, self.vp).cpu()
        # per output vector: a token whose output is small must be right too
        e = (got[..., :self.vdim] - o).norm(dim=-1) / (o.norm(dim=-1) + 0.02 * o.norm(dim=-1).mean())
        assert e.max() < tol, float(e.max())
        assert not got[..., self.vdim:].any()
        for i, s in enumerate(self.slots.tolist()):
            assert rel(self.state[s, :, :self.dim, :self.vdim].cpu(), S[i]) < tol
            assert not self.state[s, :, self.dim:].any() and not self.state[s, :, :, self.vdim:].any()
        unused = set(range(len(self.lens) + 2)) - set(self.slots.tolist())
        assert all(torch.equal(self.state[s, :, :self.dim, :self.vdim].cpu(), self.start[s]) for s in unused)
        return o, every


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("lens,H,dim,vdim,R,tau", [([1, 1, 1], 2, 40, 72, 5, 1.0), ([7, 1, 30], 3, 64, 64, 16, 16.0), ([2, 3], 1, 128, 136, 33, 4.0),
                                                   ([3, 5], 2, 200, 24, 1, 0.5), ([4, 1], 1, 300, 64, 8, 2.0)])
def test_recurrence_token_by_token(F, dtype, lens, H, dim, vdim, R, tau):
    x = Gla(F, lens, H, dim, vdim, R, tau, dtype)
    x.serial()
    o, _ = x.check(2e-5)
    F.gla_finish(x.p, x.T, x.vp, dtype == F32)
    want = oracle.rms_norm(o, x.norm, 1e-5) * torch.nn.functional.silu(x.g)
    got = x.out.view(x.T, H, x.vp).cpu()
    assert rel(got[..., :vdim], want) < (4e-3 if dtype == BF16 else 2e-5) and not got[..., vdim:].any()


# decays from mild (tau 16) to such that a block of 16 tokens leaves the range of the factored form (bias -40)
@pytest.mark.parametrize("bias,tau", [(2.0, 16.0), (0.0, 1.0), (-3.0, 1.0), (-40.0, 1.0), (-6.0, 0.1)])
@pytest.mark.parametrize("lens,H,dim,vdim,R", [([64], 2, 64, 64, 16), ([33, 100, 64, 1], 2, 40, 136, 5), ([130, 17], 1, 128, 72, 40), ([90, 32], 1, 200, 64, 8)])
def test_recurrence_in_chunks(F, lens, H, dim, vdim, R, bias, tau):
    x = Gla(F, lens, H, dim, vdim, R, tau, BF16, bias=bias, seed=dim)
    x.bias[::3] += 12.0 - bias                              # some channels hardly decay at all beside the others
    x.dev[1].copy_(_rows(x.bias.view(H, dim), x.dp).flatten())
    x.alpha = oracle.channel_decay(x.a1.double(), torch.eye(R).double(), x.a2.double(), x.bias.double(), tau).float().view(x.T, H, dim)
    x.chunked()
    x.check(2e-4)


def test_chunks_continue_a_state_and_give_snapshots(F):
    lens = [100, 150]
    a, b = Gla(F, lens, 2, 48, 80, 8, 6.0, BF16, seed=5), Gla(F, lens, 2, 48, 80, 8, 6.0, BF16, seed=5)
    rel_, idx = torch.tensor([[48, 96], [16, 112]], dtype=torch.int32).cuda(), torch.tensor([[0, 1], [2, 3]], dtype=torch.int32).cuda()
    snaps = []
    for x in (a, b):
        snap = torch.zeros(4, 2, x.dp, x.vp, device="cuda")
        x.p.snap_rel, x.p.snap_idx, x.p.snap, x.p.num_snap = rel_.data_ptr(), idx.data_ptr(), snap.data_ptr(), 2
        x.chunked([{48: 0, 96: 1}, {16: 2, 112: 3}]) if x is a else x.serial()
        _, every = x.check(2e-4)
        for e, (s, n) in enumerate([(0, 48), (0, 96), (1, 16), (1, 112)]):
            assert rel(snap[e, :, :48, :80].cpu(), every[s][n - 1]) < 2e-4
        snaps.append(snap)


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("T", [1, 5, 70, 900])
@pytest.mark.parametrize("E,identity,top,count,keep", [(1, 0, 1, 1, 1), (6, 2, 3, 4, 2), (3, 6, 2, 3, 1), (70, 10, 9, 8, 3), (257, 7, 12, 4, 4)])
def test_routing_and_permutation(F, T, E, identity, top, count, keep):
    torch.manual_seed(E + T)
    n = E + identity
    logits = torch.randn(T, n + 5, device="cuda") * 1.5
    corr = -1.5 - torch.rand(n, device="cuda")               # negative, as far apart as the scores
    valid = torch.where(torch.arange(T) % 7 == 6, -1, 3).cuda()
    ctr = F.moe_counters(300, "cuda")
    h = torch.randn(T, 128, device="cuda").to(BF16)
    want, weight = oracle.route(logits[:, :n].cpu(), torch.eye(n), corr.cpu(), {"experts": E, "identity": identity, "top": top, "groups": {"count": count, "keep": keep}})
    for f32 in (False, True):                                 # twice: the counters must be clear again
        g = F.TokenGroups(T, E, n, top, ctr, f32, "cuda")
        F.moe_route(g, logits, corr, count, keep, valid=valid)
        xs = torch.zeros(g.rows, 128, dtype=BF16, device="cuda")
        F.moe_permute(g, h, xs)
        ids, w, slot = g.ids.view(T, top).cpu(), g.weight.view(T, top).cpu(), g.slot.view(T, top).cpu()
        live = (valid >= 0).cpu()
        assert torch.equal(ids[live], want.int()[live]) and bool((ids[~live] == -1).all())
        torch.testing.assert_close(w[live], weight[live], rtol=2e-5, atol=1e-7)
        assert not ctr.any()
        used = []
        for t in range(T):
            for k in range(top):
                e, s = int(ids[t, k]), int(slot[t, k])
                assert s == (-2 if e < 0 else -1) if e < 0 or e >= E else s >= 0
                if s >= 0:
                    assert torch.equal(xs[s], h[t])
                    used.append((s, e))
        assert len({s for s, _ in used}) == len(used)
        m = int(g.num_tiles)
        tiles, expert = g.tiles[:, :m].t().tolist(), {}
        for e, r0, rows in tiles:
            assert 1 <= rows <= g.tile
            expert.update({r: e for r in range(r0, r0 + rows)})
        assert expert == dict(used)


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("T,W,E,identity,top,count,keep", [(1, 40, 1, 0, 1, 1, 1), (5, 320, 6, 2, 3, 4, 2), (64, 1500, 70, 10, 9, 8, 3), (3, 8192, 30, 2, 4, 1, 1)])
def test_norm_and_routing_in_one_kernel(F, dtype, T, W, E, identity, top, count, keep):
    """The same residual, row, choice and placed rows as the four kernels it stands for."""
    torch.manual_seed(W)
    P, n = pad64(W), E + identity
    y, x = _rows(torch.randn(T, W, device="cuda").to(dtype), P), _rows(torch.randn(T, W, device="cuda") * 3, P)
    a, b = (_rows(torch.rand(W, device="cuda") + 0.5, P) for _ in range(2))
    router = _rows((torch.randn(n, W, device="cuda") / math.sqrt(W)).to(dtype), P)
    corr, ctr = -1.0 - torch.rand(n, device="cuda"), F.moe_counters(E, "cuda")
    x2, h, h2 = x.clone(), torch.zeros(T, P, dtype=dtype, device="cuda"), torch.zeros(T, P, dtype=dtype, device="cuda")
    F.resid_norm(y, x, a, h, b, W, 1e-4)
    g = F.TokenGroups(T, E, n, top, ctr, False, "cuda", fixed=True)
    xs = torch.zeros(g.rows, P, dtype=dtype, device="cuda")
    F.moe_norm_route(y, x2, a, h2, b, W, 1e-4, g, router, corr, count, keep, xs)
    assert rel(x2, x) < 1e-6 and rel(h2, h) < 1e-3 and not ctr.any()               # sums in another order
    logits = (h2.double() @ router.double().t()).float().cpu()
    want, weight = oracle.route(logits, torch.eye(n), corr.cpu(), {"experts": E, "identity": identity, "top": top, "groups": {"count": count, "keep": keep}})
    assert torch.equal(g.ids.view(T, top).cpu(), want.int())
    torch.testing.assert_close(g.weight.view(T, top).cpu(), weight, rtol=1e-4, atol=1e-7)
    rows = [(e, r) for e, r0, k in g.tiles[:, :int(g.num_tiles)].t().tolist() for r in range(r0, r0 + k)]
    slot = g.slot.view(T, top).cpu()
    placed = [(int(want[t, k]), int(slot[t, k])) for t in range(T) for k in range(top) if want[t, k] < E]
    assert sorted(rows) == sorted(placed) and bool((slot[want >= E] == -1).all())
    assert all(torch.equal(xs[slot[t, k]], h2[t]) for t in range(T) for k in range(top) if want[t, k] < E)


@pytest.mark.parametrize("quant", ["bf16", "w8a16", "fp32"])
@pytest.mark.parametrize("T,E,top,W,ff", [(1, 5, 2, 64, 64), (40, 7, 3, 192, 128), (333, 4, 2, 128, 320), (700, 3, 2, 320, 64), (3000, 2, 2, 64, 192)])
def test_grouped_products(F, quant, T, E, top, W, ff):
    from tileinfer_b200.models.products_b200 import GroupedProduct
    torch.manual_seed(T)
    dt = F32 if quant == "fp32" else BF16
    up = [torch.randn(2 * ff, W, device="cuda") / math.sqrt(W) for _ in range(E)]
    down = [torch.randn(W, ff, device="cuda") / math.sqrt(ff) for _ in range(E)]
    g = F.TokenGroups(T, E, E, top, F.moe_counters(E, "cuda"), quant == "fp32", "cuda")
    logits = torch.randn(T, E, device="cuda")
    logits[:, 0] += 2.0                                       # a popular expert
    F.moe_route(g, logits, torch.zeros(E, device="cuda"), 1, 1)
    h = torch.randn(T, W, device="cuda").to(dt)
    xs, act = torch.zeros(g.rows, W, dtype=dt, device="cuda"), torch.zeros(g.rows, ff, dtype=dt, device="cuda")
    F.moe_permute(g, h, xs)
    GroupedProduct(up, quant, "cuda")(xs, g, None, F.GEPI_SPLIT_GLU, F.gemm_epilogue(out2=act, n_split=0, glu=(0.7, 1.702, 1.0)))
    y = torch.zeros(g.rows, W, dtype=dt, device="cuda")
    GroupedProduct(down, quant, "cuda")(act, g, y, F.GEPI_STORE)
    q8 = lambda w: gc.quantised({"x.q": w})["x.q"] if quant == "w8a16" else w.to(dt).float()
    ids, slot, tol = g.ids.view(T, top), g.slot.view(T, top), 2e-5 if quant == "fp32" else 8e-3
    x = torch.zeros(T, W, device="cuda")
    a = torch.rand(W, device="cuda") + 0.5
    want = torch.zeros(T, W, device="cuda")
    for e in range(E):
        r, k = torch.nonzero(ids == e, as_tuple=True)
        if not len(r):
            continue
        gu = h[r].float() @ q8(up[e]).t()
        gate, u = gu[:, 0::2].clamp(max=0.7), gu[:, 1::2].clamp(-0.7, 0.7)
        wa = gate * torch.sigmoid(1.702 * gate) * (u + 1)
        assert rel(act[slot[r, k].long()], wa) < tol
        wy = wa @ q8(down[e]).t()
        assert rel(y[slot[r, k].long()], wy) < 1.5 * tol
        want.index_add_(0, r, wy * g.weight.view(T, top)[r, k, None])
    hh = h.clone()
    F.resid_norm(y, x, a, hh, None, W, 1e-5, routed=g)
    assert rel(x, oracle.rms_norm(want, a, 1e-5)) < 1.5 * tol


@pytest.mark.parametrize("dtype", [BF16, F32])
def test_identity_experts_add_their_input(F, dtype):
    T, W, top = 9, 96, 3
    P = pad64(W)
    g = F.TokenGroups(T, 2, 6, top, F.moe_counters(2, "cuda"), False, "cuda")
    h, y = _rows(torch.randn(T, W, device="cuda").to(dtype), P), _rows(torch.randn(g.rows, W, device="cuda").to(dtype), P)
    g.slot.copy_(torch.randint(-2, g.rows, (T * top,)))
    g.slot[:4] = torch.tensor([-1, -1, 4, -2])
    g.weight.copy_(torch.rand(T * top))
    want = torch.zeros(T, W, device="cuda")
    for t in range(T):
        for k in range(top):
            s, a = int(g.slot[t * top + k]), float(g.weight[t * top + k])
            want[t] += a * (h[t, :W].float() if s == -1 else 0.0 if s == -2 else y[s, :W].float())
    x, one = torch.zeros(T, P, device="cuda"), _rows(torch.ones(1, W, device="cuda"), P)[0]
    hin = h.clone()
    F.resid_norm(y, x, one, h, one, W, 1e-5, routed=g)       # h is read before it is overwritten
    xs = oracle.rms_norm(want, torch.ones(W, device="cuda"), 1e-5)
    assert rel(x[:, :W], xs) < 1e-5
    assert rel(h[:, :W], oracle.rms_norm(xs, torch.ones(W, device="cuda"), 1e-5)) < (4e-3 if dtype == BF16 else 1e-5) and not torch.equal(h, hin)


# ------------------------------------------------------------------------------------------------ model against the oracle
def _want(cfg, w, toks, quant="bf16"):
    return oracle.forward(cfg, gc.quantised(w) if quant == "w8a16" else w, toks)[0]


# 32-bit: tokens choose their experts freely; 16-bit: corrections fix the choice, which a rounding could otherwise move
@pytest.mark.parametrize("quant", ["bf16", "fp32", "w8a16"])
@pytest.mark.parametrize("name", sorted(gc.CASES))
def test_whole_prompt_and_decoding(tmp_path, name, quant):
    """A whole prompt in one step, the same tokens one by one, and a long prompt followed by decoding."""
    folder, cfg, w = gc.model(tmp_path, name, decisive=quant != "fp32")
    n = 150
    t = gc.tokens(cfg, n)
    want = _want(cfg, w, t, quant)
    eng = gc.engine(folder, quant, "cuda")
    for schedule in ([[("a", n)]], gc.cut("a", n, [1]), gc.cut("a", n, [n - 20] + [1] * 20)):
        got = gc.replay(eng, schedule, {"a": t})["a"]
        gc.assert_close(got, want, quant)
    assert eng.model_runner.model.peer_status() == 0


def test_free_choice_of_experts_in_16_bit(tmp_path):
    """With free routing a rounding may swap two experts of nearly equal score: nearly all positions agree closely."""
    folder, cfg, w = gc.model(tmp_path, "groups")
    t = gc.tokens(cfg, 200)
    want = _want(cfg, w, t)
    for sizes in ([200], [50, 1]):
        got = gc.replay(gc.engine(folder, "bf16", "cuda"), gc.cut("a", 200, sizes), {"a": t})["a"]
        d = gc.errors(got, want)
        assert d.quantile(0.5) < 0.02 and d.quantile(0.9) < 0.1 and d.max() < 0.5


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
@pytest.mark.parametrize("sizes", [[2], [31], [32], [33, 2, 7], [64, 1], [100, 16, 3]])
def test_portions(tmp_path, quant, sizes):
    folder, cfg, w = gc.model(tmp_path, "mixed", decisive=quant == "bf16")
    t = gc.tokens(cfg, 237, seed=2)
    got = gc.replay(gc.engine(folder, quant, "cuda"), gc.cut("a", 237, sizes), {"a": t})["a"]
    gc.assert_close(got, _want(cfg, w, t), quant)


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
@pytest.mark.parametrize("name", ["mixed", "groups"])
def test_batches_equal_each_request_alone(tmp_path, name, quant):
    """Portions and single tokens of four requests in one step, pages and slots used again; each request gives what it
    gives alone."""
    folder, cfg, w = gc.model(tmp_path, name, decisive=quant == "bf16")
    p = {r: gc.tokens(cfg, n, seed=n) for r, n in (("a", 150), ("b", 75), ("c", 9), ("d", 130), ("e", 41), ("f", 160))}
    schedule = [[("c", 3), ("a", 100), ("b", 2)], [("b", 1), ("c", 1), ("a", 1)], [("a", 40), ("c", 5), ("b", 33)],
                [("b", 38), ("a", 9)], [("b", 1)], [("d", 64), ("e", 40), ("f", 17)],
                [("d", 1), ("e", 1), ("f", 1)], [("f", 141), ("d", 65)], [("f", 1)]]
    eng = gc.engine(folder, quant, "cuda", blocks=26)
    got = gc.replay(eng, schedule, p)
    for r, t in p.items():
        gc.assert_close(got[r], _want(cfg, w, t), quant)
        alone = gc.replay(gc.engine(folder, quant, "cuda", blocks=26, enforce_eager=True), [[(r, len(t))]], {r: t})[r]
        gc.assert_close(got[r], alone, quant)
    assert eng.scheduler.block_manager.num_free_blocks == 26 and len(eng.model_runner.free_deltanet_slots) == 4


def test_layers_on_shared_tensors_keep_their_own_cache_and_state(tmp_path):
    a = [gc.gla(2, 32, 40, 9.0), gc.attention(2, 1, 32, 40, 8)]
    cfg = gc.config(a + [gc.again(a, 1), gc.again(a, 0), gc.again(a, 1)], width=96, vocab=200)
    folder, cfg, w = gc.model(tmp_path, cfg)
    t = gc.tokens(cfg, 120)
    for quant in ("bf16", "fp32"):
        eng = gc.engine(folder, quant, "cuda")
        m = eng.model_runner.model
        assert m.layers[1] is m.layers[4] and m.layers[0] is m.layers[3] and len(m.cache) == 3 and len(m.state) == 2
        for sizes in ([120], [1], [40, 2]):
            got = gc.replay(eng, gc.cut("a", 120, sizes), {"a": t})["a"]
            gc.assert_close(got, _want(cfg, w, t), quant)


def test_far_tokens_matter(tmp_path):
    """A changed first token changes the logits hundreds of tokens later, by as much as the oracle says, in prompts and in
    decoding: through attention alone and through slowly decaying states alone."""
    sharp = gc.config([gc.attention(2, 1, 32, 40, 4, base=1e6, scale=0.6, softcap=30.0)], width=96, vocab=200)
    slow = gc.config([gc.gla(2, 32, 40, 400.0)], width=96, vocab=200)
    for k, cfg in enumerate((sharp, slow)):
        folder, cfg, w = gc.model(tmp_path / str(k), cfg)
        t = gc.tokens(cfg, 400)
        u = [(t[0] + 1) % cfg["vocab"]] + t[1:]
        change = _want(cfg, w, u) - _want(cfg, w, t)
        eng = gc.engine(folder, "fp32", "cuda")
        for sizes in ([400], [350, 1], [13]):
            d = gc.replay(eng, gc.cut("a", 400, sizes), {"a": u})["a"] - gc.replay(eng, gc.cut("a", 400, sizes), {"a": t})["a"]
            assert change[300:].abs().max() > 1e-2 and rel(d[300:], change[300:]) < 2e-2


def test_long_decoding(tmp_path):
    for quant in ("fp32", "bf16"):
        folder, cfg, w = gc.model(tmp_path / quant, "mixed", decisive=quant == "bf16")
        t = gc.tokens(cfg, 640, seed=9)
        got = gc.replay(gc.engine(folder, quant, "cuda"), gc.cut("a", 640, [2 if quant == "fp32" else 300] + [1] * 638), {"a": t})["a"]
        gc.assert_close(got, _want(cfg, w, t), quant)


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
    folder, cfg, w = gc.model(tmp_path, "mixed", decisive=quant == "bf16")
    eng = gc.engine(folder, quant, "cuda", **{"blocks": 64, **kw})
    prompts = [gc.tokens(cfg, n, seed=n) for n in (30, 90, 61, 7)]
    outs = eng.generate_token_ids(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert len(o) == 24 and _near_greedy(cfg, w, p, o, 1e-3 if quant == "fp32" else 0.2)
    if kw.get("blocks") == 16:
        assert eng.scheduler.num_preemptions > 0
    eng.close()


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
def test_prefix_reuse_restores_the_state(tmp_path, quant):
    """A cached prefix (pages and a snapshot of the states) gives the tokens that a full prefill gives."""
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = gc.model(tmp_path, "one", decisive=quant == "bf16")
    eng = gc.engine(folder, quant, "cuda", enable_prefix_caching=True)
    base, sp = gc.tokens(cfg, 130), SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    eng.generate_token_ids([base], sp)
    for n in (129, 130):
        prompt = base[:n] + gc.tokens(cfg, 21, seed=n)
        out = eng.generate_token_ids([prompt], sp)[0]
        assert _near_greedy(cfg, w, prompt, out, 1e-3 if quant == "fp32" else 0.2)
    assert eng.scheduler.prefix_cache.hit_tokens == 256


def test_sampling_with_penalties(tmp_path):
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = gc.model(tmp_path, "one")
    eng = gc.engine(folder, "bf16", "cuda")
    out = eng.generate_token_ids([gc.tokens(cfg, 70)], SamplingParams(temperature=0.8, top_k=20, repetition_penalty=1.3, max_tokens=8, ignore_eos=True))
    assert len(out[0]) == 8 and all(0 <= t < cfg["vocab"] for t in out[0])


def test_preset_with_default_settings():
    """The preset through the public API in the default (int8) mode."""
    from tileinfer_b200.engine.llm import LLM
    from tileinfer_b200.engine.sampling_params import SamplingParams
    llm = LLM("preset:tiny-gerivik", num_kvcache_blocks=64, max_num_seqs=3, max_model_len=512)
    outs = llm.generate_token_ids([list(range(1, 60)), [5, 6, 7]], SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
    assert [len(o) for o in outs] == [6, 6] and llm.model_runner.model.launches_per_decode_step > 0
    llm.close()


@pytest.mark.parametrize("dtype,quant", [("bfloat16", "bf16"), ("float32", "fp32")])
def test_trace_run(tmp_path, dtype, quant):
    folder, cfg, w = gc.model(tmp_path, "one", decisive=dtype == "bfloat16")
    t, u = gc.tokens(cfg, 60), gc.tokens(cfg, 20, seed=1)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": t[:50], "want": [49]}, {"id": "y", "tokens": u[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": u[3:], "want": [16]}, {"id": "x", "tokens": t[50:51], "want": [0]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": t[51:], "want": [8]}], "end": ["x"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens",
                        "128"], input="\n".join(map(json.dumps, lines)) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = torch.from_numpy(np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4") for i in range(3)]).reshape(4, -1))
    a, b = _want(cfg, w, t), _want(cfg, w, u)
    gc.assert_close(got, torch.stack([a[49], b[19], a[50], a[59]]), quant)
