"""Gerivik beside the framework's closest model at equal size (`python bench.py --workload gerivik`).

The closest model is the hybrid family: same width, depth and vocabulary, gated DeltaNet layers with the same state bytes in
the place of gated linear attention, attention layers of the same head count and size, and a dense feed-forward as wide as
the experts a token uses together; bf16 weights.  Random weights.  Two parts:

  throughput  prefill of one prompt (eager step) and decode steps (captured graph) of 1, 16 and 64 sequences
  kernels     every kernel of a Gerivik layer and the like kernel of the other model, on the shapes of that step: time,
              algorithmic FLOPs or bytes, and the fraction of the measured peak

CUDA events on the launching stream after warm-up.  Between timed iterations the L2 is flushed (kernels) or the step
streams more weights than it holds (throughput).
"""
from __future__ import annotations

import json
import math
import os
import sys
from dataclasses import replace

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

from benchmarks.bench_kabadra import _row, peaks, throughput, timed, timed_small  # noqa: E402

BF16 = torch.bfloat16


def closest(cfg):
    """The hybrid-family configuration of the same size."""
    from tileinfer_b200.models.config import ModelConfig
    a, g = cfg.layers[cfg.attn_layers[0]].mixer, cfg.layers[cfg.gla_layers[0]].mixer
    f = cfg.layers[0].mlp
    hv = g.heads * g.vdim // 128
    return ModelConfig(name=f"hybrid-{cfg.hidden_size}", vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, num_layers=cfg.num_layers,
                       layer_types=tuple("linear_attention" if L.is_gla else "full_attention" for L in cfg.layers),
                       intermediate_size=f.top * f.ff, num_q_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, rotary_dim=a.rot_dims,
                       rope_theta=a.rot_base, gdn_num_k_heads=hv // 2, gdn_num_v_heads=hv, gdn_head_k_dim=128, gdn_head_v_dim=128,
                       max_position_embeddings=cfg.max_position_embeddings)


class _Step:
    """A two-layer model (gla, attention) with the buffers of one step filled by running it once."""

    def __init__(self, cfg, lens, ctxs):
        from tileinfer_b200.models.gated_b200 import B200GatedModel
        from tileinfer_b200.models.gerivik import make_weights
        from tileinfer_b200.models.reference_cpu import Batch
        small = replace(cfg, layers=(cfg.layers[cfg.gla_layers[0]], cfg.layers[cfg.attn_layers[0]]))
        m = self.m = B200GatedModel(small, make_weights(small, "random:0", None, "cuda"), quant="bf16")
        per = max(ctxs) // 16 + 1
        m.alloc_cache(per * len(lens), 16, len(lens) + 1)
        for kv in m.cache.values():
            for t in kv:
                t.normal_()
        run, got = m._run_layers, []
        m._run_layers = lambda x: (got.append(x), run(x))[1]
        tables = [list(range(i * per, (i + 1) * per)) for i in range(len(lens))]
        pos = torch.cat([torch.arange(c - n, c) for n, c in zip(lens, ctxs)])
        slots = torch.cat([torch.tensor([tables[i][p // 16] * 16 + p % 16 for p in range(c - n, c)]) for i, (n, c) in enumerate(zip(lens, ctxs))])
        cu = [0]
        for n in lens:
            cu.append(cu[-1] + n)
        m.forward(Batch(torch.randint(0, small.vocab_size, (cu[-1],)), pos, cu, list(ctxs), tables, slots, list(range(len(lens)))))
        self.x = got[0]
        self.g, self.a = m.layers
        self.mg, self.ma = (L.mixer for L in small.layers)

    def bufs(self, L):
        T, x = self.x.T, self.x
        return x.proj[:T * L.n_proj].view(T, L.n_proj), x.mix[:T * L.n_mix].view(T, L.n_mix)


def kernels(cfg, prompt, ctx, batch):
    rows = kernel_rows(cfg, "prefill", [prompt], [prompt], prompt, ctx)
    torch.cuda.empty_cache()
    rows += kernel_rows(cfg, "decode", [1] * batch, [ctx] * batch, prompt, ctx)
    torch.cuda.empty_cache()
    return rows


def kernel_rows(cfg, tag, lens, ctxs, prompt, ctx):
    from tileinfer_b200.ops import functional as F
    F.L("base", "rows", "attention", "hybrid", "gla", "moe")
    s = _Step(cfg, lens, ctxs)
    m, x, W, rows = s.m, s.x, cfg.hidden_size, []
    T, S, pre = x.T, len(lens), tag == "prefill"
    small = timed if pre else timed_small
    row = lambda name, us, **kw: rows.append(_row(f"{tag}: {name}", us, **kw))
    gemm = lambda n, k, out=2: {"flops": 2 * T * n * k, "nbytes": 2 * (n * k + T * k) + out * T * n}
    lin = lambda n, k: F.LinearW(torch.randn(n, k, device="cuda").to(BF16) * k ** -0.5, False, "cuda")
    rnd = lambda *z: torch.randn(*z, device="cuda").to(BF16)
    # ---- dense products (the other model's like kernels: gate_up and down)
    mc = closest(cfg)
    kd, vd = mc.gdn_num_k_heads * 128, mc.gdn_num_v_heads * 128
    like = {"gla": (2 * kd + 2 * vd + 2 * mc.gdn_num_v_heads, vd), "attention": ((2 * mc.num_q_heads + 2 * mc.num_kv_heads) * mc.head_dim, mc.num_q_heads * mc.head_dim)}
    for name, L in (("gla", s.g), ("attention", s.a)):
        proj, mix = s.bufs(L)
        row(f"input product ({name})", timed(lambda: L.w_in(x.h, proj, F.GEPI_STORE)), **gemm(L.n_proj, W), like="input product")
        row(f"output product ({name})", timed(lambda: L.w_o(mix, x.y, F.GEPI_STORE)), **gemm(W, L.n_mix), like="output product")
        n, k = like[name]
        a, b, xa = lin(n, W), lin(W, k), rnd(T, k)
        ya, yb = torch.empty(T, n, dtype=BF16, device="cuda"), rnd(T, W)
        row(f"input product ({name}, other model)", timed(lambda: F.gemm_bf16(a, x.h, out=ya)), **gemm(n, W))
        row(f"output product ({name}, other model)", timed(lambda: F.gemm_bf16(b, xa, out=yb, epi=F.GEPI_ROWPAR, resid=yb)), **gemm(W, k, 4))
        del a, b, xa, ya, yb
    f = s.g.moe
    ff = f.top * f.ff
    up, down, act, hb = lin(2 * ff, W), lin(W, ff), rnd(T, ff), rnd(T, W)
    row("gate_up (other model)", timed(lambda: F.gemm_bf16(up, x.h, out=act, epi=F.GEPI_SWIGLU)), flops=4 * T * W * ff, nbytes=2 * (2 * ff * W + T * (W + ff)))
    row("down (other model)", timed(lambda: F.gemm_bf16(down, act, out=hb, epi=F.GEPI_ROWPAR, resid=hb)), flops=2 * T * W * ff, nbytes=2 * (ff * W + T * ff) + 4 * T * W)
    del up, down, act
    # ---- routing and experts
    L = s.g
    g = x.groups[(f.experts, f.choices, f.top)]
    n = -(-f.choices // 8) * 8
    logits = x.logits[:T * n].view(T, n)
    xs, act = x.xs[:g.rows * m.Wp].view(g.rows, m.Wp), x.act[:g.rows * L.ff].view(g.rows, L.ff)
    if g.row_stride:
        row("norm + residual + next norm + router + routing + rows to experts", small(lambda: m._norm_and_route(L, x, x.y, L.norm1b)),
            nbytes=12 * W * T + 2 * W * (f.choices + T * f.top), like="rmsnorm")
    else:
        row("router product", small(lambda: L.router(x.h, logits, F.GEPI_F32)), **gemm(f.choices, W, 4))
        row("routing", small(lambda: F.moe_route(g, logits, L.correction, f.groups, f.keep)), nbytes=T * (4 * f.choices + 12 * f.top))
        row("token rows to experts", small(lambda: F.moe_permute(g, x.h, xs)), nbytes=2 * W * T * (1 + f.top), like="rmsnorm")
        row("norm + residual + next norm", small(lambda: F.resid_norm(x.y, x.x, L.norm1b, x.h, L.norm2, W, 1e-6)), nbytes=12 * W * T, like="rmsnorm")
    live = int((g.ids < f.experts).sum())
    used = int(torch.unique(g.ids[g.ids < f.experts]).numel())
    ex = F.gemm_epilogue(out2=act, n_split=0, glu=(f.limit, 1.702, 1.0))
    row(f"experts gate/up + gated unit ({used} experts, {live} rows)", timed(lambda: L.w_up(xs, g, None, F.GEPI_SPLIT_GLU, ex)), flops=4 * live * W * L.ff,
        nbytes=2 * (used * 2 * L.ff * W + live * (W + L.ff)), like="gate_up")
    ye = torch.empty_like(xs)
    row("experts down", timed(lambda: L.w_down(act, g, ye, F.GEPI_STORE)), flops=2 * live * W * L.ff, nbytes=2 * (used * L.ff * W + live * (W + L.ff)), like="down")
    row("experts' sum + norm + residual + next norm", small(lambda: F.resid_norm(ye, x.x, L.norm2b, x.h, L.norm1, W, 1e-6, routed=g)),
        nbytes=2 * W * (live + 2 * T) + 8 * W * T, like="rmsnorm")
    nw = rnd(W)
    row("rmsnorm (other model)", small(lambda: F.rmsnorm(hb, nw, 1e-6, out=x.h)), nbytes=4 * T * W)
    # ---- gated linear attention
    proj, mix = s.bufs(s.g)
    H, dk, dv = s.mg.heads, s.mg.dim, s.mg.vdim
    io = 2 * T * (2 * H * dk + 3 * H * dv + s.g.R) + 8 * S * H * dk * dv
    state = {"flops": 4 * T * H * dk * dv, "nbytes": io}
    row("gated linear attention, all kernels", timed(lambda: m._gla(0, s.g, x, proj, mix)), **state, like="gated DeltaNet")
    if pre:
        p = m._gla_params(0, s.g, x, proj, mix)
        ck, rng = x.chunks[F.gla_chunk_size(s.g.dp)]
        p.ck_seq, p.ck_tok0, p.ck_ntok, p.ck_snap = (r.data_ptr() for r in ck)
        p.long_seq, p.long_ck, p.nc, p.num_long = x.longs.data_ptr(), rng.data_ptr(), ck.shape[1], S
        p.g_ws, p.s_ws = (w.data_ptr() for w in m.gla_ws.get(p.nc, H, dk, dv))
        row("  of it: chunk kernels", timed(lambda: F.gla_chunked(p, dk, dv)), **state)
        row("  of it: head norm + gate", timed(lambda: F.gla_finish(p, T, dv, False)), nbytes=8 * T * H * dv)
    rows.append(_like_gdn(F, tag, closest(cfg), T, S, pre))
    # ---- attention
    proj, mix = s.bufs(s.a)
    H, G, D = s.ma.heads, s.ma.kv_heads, s.ma.dim
    keys = sum(c * n - n * (n - 1) // 2 for n, c in zip(lens, ctxs))
    full = {"flops": 4 * keys * H * D, "nbytes": 2 * (T * (2 * H + 2 * G) * D + 2 * sum(ctxs) * G * D)}
    row("attention with rotation and store", timed(lambda: m._attention(1, s.a, x, proj, mix)), **full)
    prep = 2 * T * (2 * H + 4 * G) * D
    row("  of it: rotation, unit heads, store", small(lambda: m._rotate_and_store(1, s.a, x, proj)), nbytes=prep, like="qk norm")
    r, gq = F.QkvPrepParams(), rnd(T, (2 * H + 2 * G) * D)
    nw = torch.zeros(D, dtype=BF16, device="cuda")
    kc0, vc0 = (torch.zeros_like(t) for t in m.cache[1])
    qq = rnd(T, H * D)
    r.proj, r.q_norm, r.k_norm, r.positions, r.slot_mapping, r.q_out, r.kcache, r.vcache = (
        t.data_ptr() for t in (gq, nw, nw, x.positions, x.slot_mapping, qq, kc0, vc0))
    r.ld, r.hq, r.hkv, r.rotary_dim, r.eps, r.log2_theta, r.num_blocks = gq.shape[1], H, G, s.ma.rot_dims, 1e-6, math.log2(s.ma.rot_base), m.num_blocks
    row("qk norm, rotation, store (other model)", small(lambda: F.qkv_prep(r, T, D)), nbytes=prep)
    del kc0, vc0, gq, qq
    q, (kc, vc) = x.q[:T * H * D].view(T, H * D), m.cache[1]
    a = s.ma
    if pre:
        row("  of it: attention", timed(lambda: F.attn_prefill(q, kc, vc, m.num_blocks, x.block_tables, x.positions, x.tiles, None, mix, hq=H, hkv=G, D=D,
                                                              max_blocks=x.max_blocks, ld=0, scale=a.scale, softcap=a.softcap, qk_max=1.02 * D)), **full, like="attention")
        gate = rnd(T, 2 * H * D)
        row("attention (other model)", timed(lambda: F.attn_prefill(q, kc, vc, m.num_blocks, x.block_tables, x.positions, x.tiles, gate, mix, hq=H, hkv=G, D=D,
                                                                     max_blocks=x.max_blocks, ld=2 * H * D)), **full)
    else:
        p = F.AttnParams()
        p.q, p.kcache, p.vcache, p.block_tables, p.positions = (t.data_ptr() for t in (q, kc, vc, x.block_tables, x.positions))
        p.qg_seq, p.qg_tok0, p.qg_ntok, p.o_part, p.ml_part, p.out = (t.data_ptr() for t in (*x.qg, x.o_part, x.ml_part, mix))
        p.hq, p.hkv, p.rep, p.max_blocks, p.nsplit, p.num_qg, p.num_blocks = H, G, 1, x.max_blocks, x.nsplit, x.num_qg, m.num_blocks
        p.scale_log2e = a.scale * math.log2(math.e)
        p.cap_in, p.cap_out = 2 * a.scale / a.softcap * math.log2(math.e), a.softcap * math.log2(math.e)
        row("  of it: attention", timed(lambda: F.attn_paged(p, D, D)), **full, like="attention")
        gate = rnd(T, 2 * H * D)
        p.cap_out, p.gate_src, p.ld = 0.0, gate.data_ptr(), 2 * H * D
        row("attention (other model)", timed(lambda: F.attn_paged(p, D, D)), **full)
    return rows


def _like_gdn(F, tag, mc, T, S, pre):
    """The other model's recurrent layer on the same tokens."""
    hk, hv, D = mc.gdn_num_k_heads, mc.gdn_num_v_heads, 128
    kd, vd = hk * D, hv * D
    ld = (2 * kd + 2 * vd + 2 * hv + 7) // 8 * 8
    t = {"proj": torch.randn(T, ld, device="cuda").to(BF16), "conv_w": torch.randn(2 * kd + vd, 4, device="cuda"), "neg_a_exp": -torch.rand(hv, device="cuda"),
         "dt_bias": torch.randn(hv, device="cuda"), "norm_w": torch.ones(D, device="cuda"), "state": torch.zeros(S + 1, hv, D, D, device="cuda"),
         "conv_state": torch.zeros(S + 1, hv, 3, 3 * D, dtype=BF16, device="cuda"), "slots": torch.arange(S, dtype=torch.int32, device="cuda"),
         "cu": torch.arange(S + 1, dtype=torch.int32, device="cuda") * (T // S), "out": torch.zeros(T, vd, dtype=BF16, device="cuda")}
    p = F.GdnChunkParams() if pre else F.GdnParams()
    for k, v in t.items():
        setattr(p, k, v.data_ptr())
    p.ld, p.hk, p.hv, p.eps = ld, hk, hv, 1e-6
    if pre:
        ck, seq_ck = (z.cuda() for z in F.gdn_chunk_table([0, T]))
        p.ck_seq, p.ck_tok0, p.ck_ntok, p.ck_snap = (r.data_ptr() for r in ck)
        p.seq_ck, p.nc = seq_ck.data_ptr(), ck.shape[1]
        ws = F.GdnChunkWorkspace("cuda").get(p.nc * hv, D, D)
        p.wf, p.qf, p.mf, p.kf, p.u, p.gamma = (b.data_ptr() for b in ws)
        us = timed(lambda: F.gdn_chunked(p, S, T, D, D, False))
    else:
        us = timed(lambda: F.gdn_step(p, S, D, D, False, single=True))
    return _row(f"{tag}: gated DeltaNet (other model)", us, flops=6 * T * hv * D * D, nbytes=2 * T * (ld + vd) + 8 * S * hv * D * D)


def run(args) -> dict:
    from tileinfer_b200.models.gerivik import GERIVIK_2K, GERIVIK_4K
    hbm, tf, basis = peaks()
    res = {"metric": "gerivik_tok_s", "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "higher_is_better": True,
           "dtype": "bf16", "data": "synthetic: random tokens, random weights", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "basis": basis},
           "sizes": {}}
    for cfg, prompt, ctx in ((GERIVIK_2K, 8192, 2048), (GERIVIK_4K, 8192, 4096)):
        rows = kernels(cfg, prompt, ctx, 64)
        ours = throughput(cfg, prompt, ctx, (1, 16, 64), args.steps, args.warmup)
        other = throughput(closest(cfg), prompt, ctx, (1, 16, 64), args.steps, args.warmup)
        res["sizes"][cfg.name] = {"layers": cfg.num_layers, "prompt": prompt, "context": ctx, "gerivik": ours, "hybrid_model": other, "kernels": rows}
        torch.cuda.empty_cache()
    res["value"] = res["sizes"]["gerivik-4k"]["gerivik"]["decode_64_tok_s"]
    res["config"] = {"model": "gerivik-4k", "global_batch": 64, "parallelism": "tp1", "cuda_graph": True,
                     "l2": "kernels: flushed between iterations; steps: more weights than L2"}
    return res


def table(res) -> str:
    lines = []
    for name, s in res["sizes"].items():
        lines.append(f"## {name}: {s['layers']} layers, prompt {s['prompt']}, decode context {s['context']}")
        keys = [k for k in s["gerivik"]]
        lines += [f"{k:20s} gerivik {s['gerivik'][k]:>12} other {s['hybrid_model'].get(k, '-'):>12}" for k in keys]
        lines += [f"{r['us']:10.1f} us  floor {r['floor_us']:9.2f}  {r['fraction']:.3f} ({r['bound']})  {r['kernel']}" for r in s["kernels"]]
    return "\n".join(lines)


if __name__ == "__main__":
    import argparse
    ap = argparse.ArgumentParser()
    ap.add_argument("--steps", type=int, default=32)
    ap.add_argument("--warmup", type=int, default=4)
    r = run(ap.parse_args())
    print(table(r), file=sys.stderr)
    print(json.dumps(r))
