"""Luvapel on the GPU: each kernel against plain PyTorch, the model against the plain oracle in every precision, and the engine
(portions, batches, reused pages and state slots, long decoding, generation)."""
import json
import math
import os
import subprocess

import numpy as np
import pytest
import torch

import luvapel_cases as lc
import luvapel_oracle as oracle
from test_gerivik_gpu import _paged_kv, _rows, pad64, rel
from test_nogidra_gpu import _window_ref

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = torch.bfloat16, torch.float32


@pytest.fixture(scope="module")
def F():
    from tileinfer_b200.ops import functional
    functional.L("base", "rows", "attention", "conv", "delta")
    return functional


# ------------------------------------------------------------------------------------------------ row operations, products
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("two", [False, True])
@pytest.mark.parametrize("W", [40, 136, 1500, 2056, 9000])
def test_gated_residual(F, dtype, two, W):
    P, T = pad64(W), 7
    torch.manual_seed(W)
    y, z, wide = _rows(torch.randn(T, W, device="cuda"), P).to(dtype), _rows(torch.randn(T, W, device="cuda") * 5, P).to(dtype), torch.randn(T, P + 24, device="cuda").to(dtype)
    x = _rows(torch.randn(T, W, device="cuda") * 3, P)
    a, b, c = (_rows(torch.rand(W, device="cuda") + 0.5, P) for _ in range(3))
    gate, h = wide[:, 16:16 + P], torch.full((T, P), 7.0, dtype=dtype, device="cuda")
    Y = y[:, :W].float()
    if two:
        Y = 0.7 * (oracle.unit_rms(Y, 1e-3) * a[:W] + oracle.unit_rms(z[:, :W].float(), 1e-3) * b[:W])
    want = x[:, :W] + oracle.unit_rms(Y * torch.sigmoid(gate[:, :W].float()), 1e-3) * c[:W]
    F.gated_norm(y, gate, x, c, h, W, 1e-3, **(dict(y2=z, w_y=a, w_y2=b, scale=0.7) if two else {}))
    assert rel(x[:, :W], want) < 1e-6 and not x[:, W:].any()
    assert rel(h[:, :W], want) < (1e-6 if dtype == F32 else 4e-3) and not h[:, W:].any()


@pytest.mark.parametrize("dtype", [BF16, F32])
def test_embedding_in_both_precisions(F, dtype):
    W, P = 72, 128
    table, ids = _rows(torch.randn(50, W, device="cuda"), P).to(dtype), torch.tensor([3, 0, 49, 3], device="cuda")
    x, h = torch.empty(4, P, device="cuda"), torch.empty(4, P, dtype=dtype, device="cuda")
    F.embed_pos(ids, torch.zeros(4, dtype=torch.int32, device="cuda"), table, None, None, x, W, 1e-6, scale=2.5, h=h)
    want = table[ids].float() * 2.5
    assert torch.equal(x, want) and torch.equal(h, want.to(dtype))


@pytest.mark.parametrize("quant", ["bf16", "w8a16", "fp32"])
@pytest.mark.parametrize("M,N,K,split", [(1, 64, 64, 0), (5, 192, 4160, 64), (40, 200, 192, 192), (130, 328, 192, 8), (700, 4096, 256, 2048)])
def test_squared_positive_part(F, quant, M, N, K, split):
    from tileinfer_b200.models.products_b200 import Product
    torch.manual_seed(N)
    dt = F32 if quant == "fp32" else BF16
    w, x, b = torch.randn(N, K, device="cuda").to(BF16) / K ** 0.5, torch.randn(M, K, device="cuda").to(dt), torch.randn(N, device="cuda")
    P = Product(w, quant, "cuda")
    dense = w.float() if quant != "w8a16" else P.w.dense().float()
    y = x.float() @ dense.T + b
    out, act = torch.full((M, max(split, 8)), 7.0, dtype=dt, device="cuda"), torch.empty(M, N - split, dtype=dt, device="cuda")
    P(x, out, F.GEPI_SPLIT_RELU2, F.gemm_epilogue(out2=act, n_split=split, bias=b))
    tol = 1e-5 if quant == "fp32" else 8e-3
    assert rel(act, y[:, split:].clamp(min=0) ** 2) < tol
    assert rel(out[:, :split], y[:, :split]) < tol if split else (out == 7).all()


# ------------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,G,dim,dp,rot", [(3, 1, 24, 64, 18), (4, 2, 64, 64, 64), (2, 2, 100, 128, 2), (1, 1, 300, 320, 0), (34, 2, 128, 128, 40)])
def test_heads_normed_one_by_one(F, dtype, H, G, dim, dp, rot):
    """Weights per head (a temperature is part of them), rotation in neighbouring pairs, and the keys as projected as values."""
    torch.manual_seed(dim)
    T, nb, ld = 6, 4, (H + G) * dp + 8
    q, k = (torch.randn(T, a, dim, device="cuda").to(dtype) for a in (H, G))
    qw, kw = torch.rand(H, dim, device="cuda") + 0.5, torch.rand(G, dim, device="cuda") + 0.5
    proj = torch.zeros(T, ld, dtype=dtype, device="cuda")
    proj[:, :(H + G) * dp] = torch.cat([_rows(q, dp), _rows(k, dp)], 1).flatten(1)
    pos = torch.tensor([0, 1, 17, 1000, 3000, 5], dtype=torch.int32, device="cuda")
    slots = torch.tensor([5, 16, -1, 63, 64, 33], device="cuda")                   # -1 and 64 are not in the cache
    inv = torch.tensor([900.0 ** (-2 * i / rot) for i in range(rot // 2)] or [0.0], dtype=torch.float64).float().cuda()
    qo, kc, vc = torch.zeros(T, H, dp, dtype=dtype, device="cuda"), torch.zeros(nb, G, 16, dp, dtype=dtype, device="cuda"), \
        torch.zeros(nb, G, dp, 16, dtype=dtype, device="cuda")
    qwp, kwp = _rows(qw, dp).flatten().contiguous(), _rows(kw, dp).flatten().contiguous()
    p = F.RopeUnitParams()
    p.proj, p.q_w, p.k_w, p.inv_freq, p.positions = proj.data_ptr(), qwp.data_ptr(), kwp.data_ptr(), inv.data_ptr(), pos.data_ptr()
    p.slot_mapping, p.q_out, p.kcache, p.vcache = slots.data_ptr(), qo.data_ptr(), kc.data_ptr(), vc.data_ptr()
    p.T, p.ld, p.q_col, p.k_col, p.v_col, p.H, p.G = T, ld, 0, H * dp, H * dp, H, G
    p.dim, p.dp, p.vp, p.half, p.num_blocks, p.eps, p.pairs = dim, dp, dp, rot // 2, nb, 1e-4, 1
    F.rope_unit(p, dtype == F32)
    turn = lambda x, w: oracle.rotate_pairs((oracle.unit_rms(x.double(), 1e-4) * w.double()).cpu(), pos.cpu(), 900.0, rot).cuda()
    tol = 4e-3 if dtype == BF16 else 2e-4                                           # 32-bit angles of 3000 radians
    assert rel(qo[..., :dim], turn(q, qw)) < tol and not qo[..., dim:].any()
    kwant, vwant = torch.zeros(nb * 16, G, dp, device="cuda"), torch.zeros(nb * 16, G, dp, device="cuda")
    for t in (0, 1, 3, 5):
        kwant[slots[t], :, :dim], vwant[slots[t], :, :dim] = turn(k, kw)[t].float(), k[t].float()
    assert rel(kc.permute(0, 2, 1, 3).reshape(nb * 16, G, dp), kwant) < tol
    assert torch.equal(vc.permute(0, 3, 1, 2).reshape(nb * 16, G, dp).float(), vwant)


@pytest.mark.parametrize("H,G,d,window,nsplit", [(2, 1, 64, 17, 3), (6, 2, 128, 100, 2), (3, 3, 256, 300, 1), (34, 2, 64, 1, 2)])
def test_gates_per_output_dimension(F, H, G, d, window, nsplit):
    """The paged, the tiled and the plain attention read gates at any column and pitch."""
    torch.manual_seed(H + d)
    n, scale = 300, 1.5 / math.sqrt(d)
    q, k, v = (torch.randn(n, a, d, device="cuda").to(BF16) for a in (H, G, G))
    gate = torch.randn(n, 16 + H * d + 8, device="cuda").to(BF16)
    kc, vc, table = _paged_kv(k, v, G)
    pos = torch.arange(n, dtype=torch.int32, device="cuda")
    want = _window_ref(q, k, v, pos, scale, window) * torch.sigmoid(gate[:, 16:16 + H * d].float()).view(n, H, d)
    out = torch.zeros(n, H * d + 64, dtype=BF16, device="cuda")
    tiles = torch.tensor([(0, a, min(128, n - a)) for a in range(0, n, 128)], dtype=torch.int32).t().contiguous().cuda()
    F.attn_prefill(q, kc, vc, kc.shape[0], table, pos, tiles, gate, out, hq=H, hkv=G, D=d, max_blocks=table.shape[1], ld=gate.stride(0), scale=scale,
                   window=window, gate_col=16, gate_stride=d)
    assert rel(out[:, :H * d].view(n, H, d), want) < 6e-3 and not out[:, H * d:].any()
    rows = [0, 1, 16, 63, 130, 255, 299]
    idx = torch.tensor(rows, device="cuda")
    tok, one, zero = idx.int(), torch.ones(len(rows), dtype=torch.int32, device="cuda"), torch.zeros(len(rows), dtype=torch.int32, device="cuda")
    for dtype, general in ((BF16, False), (BF16, True), (F32, True)):
        a = F.AttnGeneralParams() if general else F.AttnParams()
        Q, K, V, Gt, out = q.to(dtype), kc.to(dtype), vc.to(dtype), gate.to(dtype), torch.zeros(n, H * d, dtype=dtype, device="cuda")
        a.q, a.kcache, a.vcache, a.out = Q.data_ptr(), K.data_ptr(), V.data_ptr(), out.data_ptr()
        a.block_tables, a.positions, a.qg_seq, a.qg_tok0, a.qg_ntok = table.data_ptr(), pos.data_ptr(), zero.data_ptr(), tok.data_ptr(), one.data_ptr()
        a.max_blocks, a.num_qg, a.num_blocks, a.ldo, a.window = table.shape[1], len(rows), kc.shape[0], H * d, window
        if general:
            a.H, a.G, a.dp, a.vp, a.scale, a.gate, a.ldg, a.gcol = H, G, d, d, scale, Gt.data_ptr(), Gt.stride(0), 16
            F.attn_general(a, dtype == F32)
        else:
            per = H // G
            a.rep = per // max(x for x in range(1, 17) if per % x == 0)
            a.hq, a.hkv, a.nsplit, a.scale_log2e = H, G, nsplit, scale * math.log2(math.e)
            o = torch.empty(len(rows) * G * a.rep * nsplit * 16 * d, device="cuda")
            ml = torch.empty(len(rows) * G * a.rep * nsplit * 32, device="cuda")
            a.o_part, a.ml_part = o.data_ptr(), ml.data_ptr()
            a.gate_src, a.ld, a.gate_col, a.gate_stride = Gt.data_ptr(), Gt.stride(0), 16, d
            F.attn_paged(a, d, d)
        torch.cuda.synchronize()
        assert rel(out[idx].view(-1, H, d), want[idx]) < (6e-3 if dtype == BF16 else 2e-5)


# ------------------------------------------------------------------------------------------------ delta rules
KEY_SIZES = (64, 128, 256, 512)


class Delta:
    """Inputs of the delta-rule kernels for sequences of the given lengths, and what the plain recurrences make of them in 64-bit."""

    def __init__(self, F, dtype, general, H, G, D, V, R, lens, seed=0, decay=0.0, one_key=False):
        g = torch.Generator().manual_seed(seed)
        rnd = lambda *s: torch.randn(*s, generator=g)
        self.F, self.dtype, self.general, self.lens, T = F, dtype, general, lens, sum(lens)
        self.cu = [sum(lens[:i]) for i in range(len(lens) + 1)]
        self.H, self.G, self.D, self.V, self.dk, self.dv = H, G, D, V, next(s for s in KEY_SIZES if s >= D), pad64(V)
        q, k, v = (t.to(dtype).double() for t in (rnd(T, G, D), rnd(T, G, D), rnd(T, H, V)))
        if one_key:                                          # every token with nearly the same key: reads chain through a chunk
            k = (k[:1] + 0.1 * k).to(dtype).double()
        self.slots = torch.tensor([len(lens) - s for s in range(len(lens))], dtype=torch.int32)
        S0 = rnd(len(lens) + 2, H, D, V).double()
        self.S0, self.o, self.states = S0, torch.zeros(T, H, V, dtype=torch.float64), S0.clone()
        pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1])).flatten(-2)
        heads = torch.cat([pad(q, self.dk), pad(k, self.dk), pad(v, self.dv)], 1)
        p = self.p = F.DeltaParams()
        if general:
            a, x, w2, w0, bias = rnd(T, H, D).to(dtype).double() + decay, rnd(T, R).to(dtype).double(), rnd(R, H, D).double() / R ** 0.5, rnd(H, D).double() + decay, rnd(H, D).double()
            w0, w2, bias, a = w0.float().double(), w2.float().double(), bias.float().double(), a.to(dtype).double()
            z = (torch.tanh(x) @ w2.flatten(1)).view(T, H, D) + w0
            self.rule = ((-math.exp(-0.5) * torch.sigmoid(z)).exp(), torch.sigmoid(a + bias))
            cols = torch.cat([heads, pad(a, self.dk), x, torch.zeros(T, -R % 8)], 1)
            self.src = self.proj = cols.to(dtype).cuda()
            keep = [pad(bias, self.dk), pad(w0, self.dk), pad(w2, self.dk)]
            self.keep = [t.float().contiguous().cuda() for t in keep]
            p.bias, p.w0, p.w2 = (t.data_ptr() for t in self.keep)
            p.b_col, p.a_col, p.R, p.decay_scale, p.q_scale = heads.shape[1], heads.shape[1] + H * self.dk, R, math.exp(-0.5), 1.0
        else:
            A, dt, b, a = (rnd(H) * 0.5 + decay).float().double(), (rnd(H) * 0.5).float().double(), rnd(T, H).to(dtype).double(), rnd(T, H).to(dtype).double()
            self.rule = (torch.exp(-torch.exp(A) * oracle.softplus(a + dt)), torch.sigmoid(b))
            q, k = oracle.unit_length(q) * D ** -0.5, oracle.unit_length(k)
            self.src, self.proj = heads.to(dtype).cuda(), torch.cat([torch.zeros(T, 8), b, torch.zeros(T, -H % 8), a, torch.zeros(T, -H % 8)], 1).to(dtype).cuda()
            self.keep = [t.float().cuda() for t in (dt, -torch.exp(A))]
            p.bias, p.neg_a = (t.data_ptr() for t in self.keep)
            p.b_col, p.a_col, p.q_scale = 8, 8 + H + -H % 8, D ** -0.5
        self.qkv = (q, k, v)
        for s in range(len(lens)):
            for h in range(H):
                self.o[self.cu[s]:self.cu[s + 1], h], self.states[self.slots[s], h] = self.run(s, h, lens[s])
        self.state = torch.nn.functional.pad(S0, (0, self.dv - V, 0, self.dk - D)).float().cuda().contiguous()
        self.out, self.d_slots, self.d_cu = torch.full((T, H, self.dv), 7.0, device="cuda"), self.slots.cuda(), torch.tensor(self.cu, dtype=torch.int32).cuda()
        p.src, p.proj, p.state, p.slots, p.cu, p.o = (t.data_ptr() for t in (self.src, self.proj, self.state, self.d_slots, self.d_cu, self.out))
        p.lds, p.ld, p.H, p.rep = self.src.stride(0), self.proj.stride(0), H, H // G
        p.q_col, p.k_col, p.v_col = 0, G * self.dk, 2 * G * self.dk

    def run(self, s, h, n):
        """(outputs, state) of head h after n tokens of sequence s."""
        at, kh, S0 = slice(self.cu[s], self.cu[s] + n), h // (self.H // self.G), self.S0[self.slots[s], h].float().double()
        q, k, v = self.qkv[0][at, kh], self.qkv[1][at, kh], self.qkv[2][at, h]
        a, b = self.rule[0][at, h], self.rule[1][at, h]
        return oracle.general_delta_rule(q, k, v, a, b, S0) if self.general else oracle.delta_rule(q, k, v, a, b, S0)

    def step(self, seqs=None):
        n = len(self.lens)
        if seqs is not None:
            self._seqs, n = torch.tensor(seqs, dtype=torch.int32).cuda(), len(seqs)
            self.p.seqs = self._seqs.data_ptr()
        self.F.delta_step(self.p, n, self.dk, self.dv, self.general, self.dtype == F32)

    def chunked(self, seqs, points=None):
        ck, rng = self.F.gla_chunk_table(self.cu, seqs, self.F.delta_chunk_size(self.dk), points)
        self._ck, self._rng, self._long = ck.cuda(), rng.cuda(), torch.tensor(seqs, dtype=torch.int32).cuda()
        p = self.p
        p.ck_seq, p.ck_tok0, p.ck_ntok, p.ck_snap = (r.data_ptr() for r in self._ck)
        p.long_seq, p.long_ck, p.nc, p.num_long = self._long.data_ptr(), self._rng.data_ptr(), ck.shape[1], len(seqs)
        self._ws = self.F.DeltaWorkspace("cuda")
        p.t_ws, p.q_ws, p.s_ws, p.f_ws = (w.data_ptr() for w in self._ws.get(p.nc, self.H, self.dk, self.dv))
        self.F.delta_chunked(p, self.dk, self.dv, self.general)

    def check(self, tol):
        torch.cuda.synchronize()
        D, V = self.D, self.V
        assert rel(self.out[..., :V], self.o.cuda()) < tol and not self.out[..., V:].any()
        assert rel(self.state[..., :D, :V], self.states.cuda()) < tol and not self.state[..., V:].any() and not self.state[..., D:, :].any()
        heads = (self.out[..., :V].double() - self.o.cuda()).norm(dim=-1) / self.o.cuda().norm(dim=-1).clamp_min(1e-3)
        assert heads.quantile(0.99) < 10 * tol


GATED = [(False, 4, 2, 24, 40, 0), (False, 3, 3, 64, 64, 0), (False, 6, 2, 130, 130, 0), (False, 2, 1, 128, 256, 0), (False, 2, 2, 40, 20, 0)]
GENERAL = [(True, 3, 3, 24, 24, 5), (True, 2, 2, 64, 64, 16), (True, 2, 2, 128, 128, 40), (True, 1, 1, 200, 200, 33)]
BEYOND = [(False, 2, 1, 300, 24, 0), (True, 1, 1, 270, 270, 7)]


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("general,H,G,D,V,R", GATED + GENERAL + BEYOND)
def test_delta_rules_token_by_token(F, dtype, general, H, G, D, V, R):
    x = Delta(F, dtype, general, H, G, D, V, R, [1, 5, 33, 2])
    x.step()
    x.check(1e-5)
    one = Delta(F, dtype, general, H, G, D, V, R, [1, 1, 1], seed=1)
    one.p.cu = 0                                             # the decode form
    one.step()
    one.check(1e-5)


# weak decay (states of hundreds of tokens), the usual, and strong
@pytest.mark.parametrize("decay", [-5.0, 0.0, 3.0])
@pytest.mark.parametrize("general,H,G,D,V,R", GATED + GENERAL)
def test_delta_rules_in_chunks(F, general, H, G, D, V, R, decay):
    x = Delta(F, BF16, general, H, G, D, V, R, [64, 3, 200, 65, 1, 63], decay=decay)
    x.chunked([0, 2, 3, 5])
    x.step([1, 4])
    x.check(3e-4)


@pytest.mark.parametrize("general,H,G,D,V,R", [GATED[1], GENERAL[1], GENERAL[2]])
def test_delta_rules_with_one_key_again_and_again(F, general, H, G, D, V, R):
    """Every token reads what the one before it wrote: the triangular system of a chunk is far from the identity."""
    for decay in (-4.0, 1.0):
        x = Delta(F, BF16, general, H, G, D, V, R, [130, 70], decay=decay, one_key=True)
        x.chunked([0, 1])
        x.check(3e-4)


@pytest.mark.parametrize("general,H,G,D,V,R", [GATED[0], GENERAL[0]])
@pytest.mark.parametrize("chunked", [True, False])
def test_delta_rule_snapshots(F, general, H, G, D, V, R, chunked):
    x = Delta(F, BF16, general, H, G, D, V, R, [150, 40], seed=4)
    snap = torch.zeros(3, H, x.dk, x.dv, device="cuda")
    points = [{48: 0, 128: 2}, {32: 1}]
    rel_, idx = torch.tensor([[48, 128], [32, 0]], dtype=torch.int32).cuda(), torch.tensor([[0, 2], [1, 0]], dtype=torch.int32).cuda()
    x.p.snap_rel, x.p.snap_idx, x.p.snap, x.p.num_snap = rel_.data_ptr(), idx.data_ptr(), snap.data_ptr(), 2
    x.chunked([0, 1], points) if chunked else x.step()
    x.check(3e-4)
    for e, s, n in ((0, 0, 48), (2, 0, 128), (1, 1, 32)):
        for h in range(H):
            assert rel(snap[e, h, :D, :V], x.run(s, h, n)[1].cuda()) < 3e-4


@pytest.mark.parametrize("dtype", [BF16, F32])
@pytest.mark.parametrize("H,V,silu", [(3, 20, True), (2, 64, False), (5, 200, False), (1, 300, True)])
def test_head_norm_and_gate(F, dtype, H, V, silu):
    T, dv = 5, pad64(V)
    o, w = _rows(torch.randn(T, H, V, device="cuda"), dv), torch.rand(H, V, device="cuda") + 0.5
    gate = torch.randn(T, 16 + H * dv, device="cuda").to(dtype)
    for per_head in (False, True):
        norm = _rows(w, dv) if per_head else _rows(w[0], dv)
        out = torch.full((T, H * dv + 16), 7.0, dtype=dtype, device="cuda")
        F.head_norm(o, gate, 16, norm, out, V, 1e-4, silu)
        z = gate[:, 16:].float().view(T, H, dv)[..., :V]
        want = oracle.unit_rms(o[..., :V], 1e-4) * (w if per_head else w[0]) * torch.sigmoid(z) * (z if silu else 1.0)
        got = out[:, :H * dv].view(T, H, dv)
        assert rel(got[..., :V], want) < (4e-3 if dtype == BF16 else 1e-6) and not got[..., V:].any() and (out[:, H * dv:] == 7).all()


# ------------------------------------------------------------------------------------------------ model
def _want(cfg, w, toks):
    return oracle.forward(cfg, w, toks)[0]


@pytest.mark.parametrize("quant", ["fp32", "bf16", "w8a16"])
@pytest.mark.parametrize("name", sorted(lc.CASES))
def test_prompts_and_decoding_match_oracle(tmp_path, name, quant):
    """Whole prompts, and the same tokens one by one, against the plain equations."""
    folder, cfg, w = lc.model(tmp_path, name)
    t = lc.tokens(cfg, 211)
    want = _want(cfg, lc.quantised(w) if quant == "w8a16" else w, t)
    eng = lc.engine(folder, quant, "cuda")
    for sizes in ([211], [150, 1]):
        lc.assert_close(lc.replay(eng, lc.cut("a", 211, sizes), {"a": t})["a"], want, quant)
    lc.assert_close(lc.replay(eng, lc.cut("a", 40, [1]), {"a": t[:40]})["a"], want[:40], quant)
    eng.close()


def test_residual_stream_layer_by_layer(tmp_path):
    """The residual after every layer: the model cut off behind it."""
    folder, cfg, w = lc.model(tmp_path, "mixed")
    t = lc.tokens(cfg, 60)
    stream = oracle.forward(cfg, w, t)[1]
    from tileinfer_b200.models.checkpoint import CheckpointWeights
    from tileinfer_b200.models.delta_b200 import B200DeltaModel
    from tileinfer_b200.models.luvapel import LuvapelConfig
    from tileinfer_b200.models.reference_cpu import Batch
    rank = {i: lc.RANKS["mixed"] for i in range(len(cfg["layers"]))}
    for n in range(1, len(cfg["layers"]) + 1):
        mc = LuvapelConfig.from_dict(dict(cfg, layers=cfg["layers"][:n]), decay_rank=rank)
        m = B200DeltaModel(mc, CheckpointWeights(mc, folder), quant="fp32")
        m.alloc_cache(8, 16, 2)
        b = Batch(torch.tensor(t), torch.arange(60), [0, 60], [60], [[5, 2, 7, 0]], torch.tensor([[5, 2, 7, 0][j // 16] * 16 + j % 16 for j in range(60)]),
                  [1], out_rows=list(range(60)))
        assert rel(m.forward(b)[:, :cfg["width"]].cpu(), stream[n - 1]) < 1e-5


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
@pytest.mark.parametrize("sizes", [[2], [31], [32], [33, 2, 7], [64, 1], [100, 16, 3]])
def test_portions(tmp_path, quant, sizes):
    folder, cfg, w = lc.model(tmp_path, "mixed")
    t = lc.tokens(cfg, 237, seed=2)
    got = lc.replay(lc.engine(folder, quant, "cuda"), lc.cut("a", 237, sizes), {"a": t})["a"]
    lc.assert_close(got, _want(cfg, w, t), quant)


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_batches_equal_each_request_alone(tmp_path, name, quant):
    """Portions and single tokens of four requests in one step, pages and slots used again; each request gives what it
    gives alone."""
    folder, cfg, w = lc.model(tmp_path, name)
    p = {r: lc.tokens(cfg, n, seed=n) for r, n in (("a", 150), ("b", 75), ("c", 9), ("d", 130), ("e", 41), ("f", 160))}
    schedule = [[("c", 3), ("a", 100), ("b", 2)], [("b", 1), ("c", 1), ("a", 1)], [("a", 40), ("c", 5), ("b", 33)],
                [("b", 38), ("a", 9)], [("b", 1)], [("d", 64), ("e", 40), ("f", 17)],
                [("d", 1), ("e", 1), ("f", 1)], [("f", 141), ("d", 65)], [("f", 1)]]
    eng = lc.engine(folder, quant, "cuda", blocks=26)
    got = lc.replay(eng, schedule, p)
    for r, t in p.items():
        lc.assert_close(got[r], _want(cfg, w, t), quant)
        alone = lc.replay(lc.engine(folder, quant, "cuda", blocks=26, enforce_eager=True), [[(r, len(t))]], {r: t})[r]
        lc.assert_close(got[r], alone, quant)
    assert eng.scheduler.block_manager.num_free_blocks == 26 and len(eng.model_runner.free_deltanet_slots) == 4


@pytest.mark.parametrize("window", [1, 16, 33, 129])
def test_what_a_token_reaches(tmp_path, window):
    """One layer whose recurrent half is switched off, one changed token: the logits change for exactly as many tokens as the
    window reaches, in prompts and in decoding, and by as much as the oracle says."""
    cfg = lc.config([lc.parallel(lc.attention(2, 1, 24, 24, window), lc.gated(1, 1, 8, 8, 2))], width=96, vocab=200)
    w = oracle.random_weights(cfg, 3)
    w["l0.mix.right.out"] = torch.zeros_like(w["l0.mix.right.out"])
    folder = oracle.write_model(str(tmp_path / "m"), cfg, w)
    t, at = lc.tokens(cfg, 180), 21
    u = t[:at] + [(t[at] + 1) % cfg["vocab"]] + t[at + 1:]
    change = _want(cfg, w, u) - _want(cfg, w, t)
    reach = at + window
    assert change[at:reach].abs().amax(-1).min() > 1e-6 and not change[reach:].any()
    eng = lc.engine(folder, "fp32", "cuda")
    for sizes in ([180], [60, 1], [13]):
        d = lc.replay(eng, lc.cut("a", 180, sizes), {"a": u})["a"] - lc.replay(eng, lc.cut("a", 180, sizes), {"a": t})["a"]
        assert rel(d, change) < 1e-2 and not d[:at].any() and not d[reach:].any()


@pytest.mark.parametrize("window,key", [(40, 16), (129, 127), (200, 31), (17, 300)])
def test_window_edge_of_one_key_that_stands_out(tmp_path, window, key):
    """One token's key meets every query with a score far above the others: it is seen while it is window - 1 tokens back and
    no longer one token on, in prompts, portions and decoding, in 16 and in 32 bits."""
    cfg = lc.config([lc.parallel(lc.attention(2, 1, 24, 0, window), lc.gated(1, 1, 8, 8, 2))], width=96, vocab=200, scale=1.0)
    w = oracle.random_weights(cfg, 3)
    w["l0.mix.right.out"] = torch.zeros_like(w["l0.mix.right.out"])
    # channel 0 of the residual is 0.1 for every token but the marked one (id 7: 8); queries point at what its key is made of
    w["embed"][:, 0], w["embed"][7, 0] = 0.1, 8.0
    for head in range(2):
        w["l0.mix.left.q"][head * 24, :], w["l0.mix.left.q"][head * 24, 0] = 0.0, 100.0
    w["l0.mix.left.k"][0, :], w["l0.mix.left.k"][0, 0] = 0.0, 10.0
    w["l0.mix.left.temp"][:] = 3.0
    folder = oracle.write_model(str(tmp_path / "m"), cfg, w)
    t = [x if x != 7 else 8 for x in lc.tokens(cfg, 340)]
    t[key] = 7
    want = _want(cfg, w, t)
    last = min(340, key + window) - 1
    if last + 1 < 340:                                       # the edge shows
        assert (want[last] - want[last + 1]).norm() > 0.1 * want[last].norm()
    for quant in ("fp32", "bf16"):
        eng = lc.engine(folder, quant, "cuda")
        for sizes in ([340], [64, 2], [300, 1]):
            lc.assert_close(lc.replay(eng, lc.cut("a", 340, sizes), {"a": t})["a"], want, quant)


@pytest.mark.parametrize("kind", ["parallel", "general"])
def test_slow_states_carry_the_first_token(tmp_path, kind):
    """With hardly any decay a changed first token changes the logits hundreds of tokens later, by as much as the oracle says."""
    layer = lc.general(2, 40) if kind == "general" else lc.parallel(lc.attention(1, 1, 16, 16, 4), lc.gated(2, 1, 64, 24, 4))
    cfg = lc.config([layer], width=96, vocab=200)
    w = oracle.random_weights(cfg, 3)
    if kind == "general":
        w["l0.mix.w0"], w["l0.mix.a.b"] = torch.full_like(w["l0.mix.w0"], -8.0), torch.full_like(w["l0.mix.a.b"], -6.0)
        for n in ("l0.mix.a", "l0.mix.w2"):
            w[n] = (0.02 * w[n].float()).to(BF16)
    else:
        # steps are small wherever channel 0 of the embedding is one, which is everywhere but at the first token
        w["l0.mix.right.A_log"], w["l0.mix.left.out"] = torch.full_like(w["l0.mix.right.A_log"], -7.0), torch.zeros_like(w["l0.mix.left.out"])
        w["embed"][:, 0], w["embed"][:2, 0], w["l0.mix.right.b"][:, 0] = 1.0, -1.0, -0.4
    w["embed"][:2] *= 8                                     # the first token writes more than the others
    folder = oracle.write_model(str(tmp_path / "m"), cfg, w)
    t = [0] + [max(2, x) for x in lc.tokens(cfg, 399)]
    u = [1] + t[1:]
    change = _want(cfg, w, u) - _want(cfg, w, t)
    assert change[300:].abs().max() > 0.1
    for quant, tol in (("fp32", 2e-2), ("bf16", 0.5)):
        eng = lc.engine(folder, quant, "cuda")
        for sizes in ([400], [350, 1], [70]):
            d = lc.replay(eng, lc.cut("a", 400, sizes), {"a": u})["a"] - lc.replay(eng, lc.cut("a", 400, sizes), {"a": t})["a"]
            assert rel(d[300:], change[300:]) < tol


def test_long_decoding(tmp_path):
    folder, cfg, w = lc.model(tmp_path, "mixed")
    t = lc.tokens(cfg, 640, seed=9)
    want = _want(cfg, w, t)
    for quant in ("fp32", "bf16"):
        got = lc.replay(lc.engine(folder, quant, "cuda"), lc.cut("a", 640, [2 if quant == "fp32" else 300] + [1] * 638), {"a": t})["a"]
        lc.assert_close(got, want, quant)


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
    folder, cfg, w = lc.model(tmp_path, "mixed")
    eng = lc.engine(folder, quant, "cuda", **{"blocks": 64, **kw})
    prompts = [lc.tokens(cfg, n, seed=n) for n in (30, 90, 61, 7)]
    outs = eng.generate_token_ids(prompts, SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert len(o) == 24 and _near_greedy(cfg, w, p, o, 1e-3 if quant == "fp32" else 0.2)
    if kw.get("blocks") == 16:
        assert eng.scheduler.num_preemptions > 0
    eng.close()


@pytest.mark.parametrize("quant", ["bf16", "fp32"])
@pytest.mark.parametrize("name", ["one", "recurrent"])
def test_prefix_reuse(tmp_path, name, quant):
    """A cached prefix (pages, and a snapshot of states and convolution inputs) gives the tokens that a full prefill gives."""
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = lc.model(tmp_path, name)
    eng = lc.engine(folder, quant, "cuda", enable_prefix_caching=True)
    base, sp = lc.tokens(cfg, 130), SamplingParams(temperature=0.0, max_tokens=8, ignore_eos=True)
    eng.generate_token_ids([base], sp)
    for n in (129, 130):
        prompt = base[:n] + lc.tokens(cfg, 21, seed=n)
        out = eng.generate_token_ids([prompt], sp)[0]
        assert _near_greedy(cfg, w, prompt, out, 1e-3 if quant == "fp32" else 0.2)
    assert eng.scheduler.prefix_cache.hit_tokens == 256


def test_sampling_with_penalties(tmp_path):
    from tileinfer_b200.engine.sampling_params import SamplingParams
    folder, cfg, w = lc.model(tmp_path, "one")
    eng = lc.engine(folder, "bf16", "cuda")
    out = eng.generate_token_ids([lc.tokens(cfg, 70)], SamplingParams(temperature=0.8, top_k=20, repetition_penalty=1.3, max_tokens=8, ignore_eos=True))
    assert len(out[0]) == 8 and all(0 <= t < cfg["vocab"] for t in out[0])


def test_preset_with_default_settings():
    """The preset through the public API in the default (int8) mode."""
    from tileinfer_b200.engine.llm import LLM
    from tileinfer_b200.engine.sampling_params import SamplingParams
    llm = LLM("preset:tiny-luvapel", num_kvcache_blocks=64, max_num_seqs=3, max_model_len=512)
    outs = llm.generate_token_ids([list(range(1, 60)), [5, 6, 7]], SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
    assert [len(o) for o in outs] == [6, 6] and llm.model_runner.model.launches_per_decode_step > 0
    llm.close()


@pytest.mark.parametrize("dtype,quant", [("bfloat16", "bf16"), ("float32", "fp32")])
def test_trace_run(tmp_path, dtype, quant):
    folder, cfg, w = lc.model(tmp_path, "one")
    t, u = lc.tokens(cfg, 60), lc.tokens(cfg, 20, seed=1)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": t[:50], "want": [49]}, {"id": "y", "tokens": u[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": u[3:], "want": [16]}, {"id": "x", "tokens": t[50:51], "want": [0]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": t[51:], "want": [8]}], "end": ["x"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens",
                        "128"], input="\n".join(map(json.dumps, lines)) + "\n", capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = torch.from_numpy(np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4") for i in range(3)]).reshape(4, -1))
    a, b = _want(cfg, w, t), _want(cfg, w, u)
    lc.assert_close(got, torch.stack([a[49], b[19], a[50], a[59]]), quant)
