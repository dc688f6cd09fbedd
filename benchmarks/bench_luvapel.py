"""Luvapel beside the framework's closest model at equal size (`python bench.py --workload luvapel`).

The closest model is the hybrid family: same width, depth and vocabulary, gated DeltaNet layers with the same state bytes where
Luvapel has a general delta rule, gated attention layers of the same heads where it has a parallel mixer, and a gated
feed-forward with as many weights as the squared one; bf16 weights.  Random weights.  Two parts:

  throughput  prefill of one prompt (eager step) and decode steps (captured graph) of 1, 16 and 64 sequences
  kernels     every kernel of Luvapel's layers and the like kernel of the hybrid model (of Gerivik for the residual's row
              operations), on the shapes of that step: time, algorithmic FLOPs or bytes, and the fraction of the measured peak

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

from benchmarks.bench_gerivik import _like_gdn  # noqa: E402
from benchmarks.bench_kabadra import _row, peaks, throughput, timed, timed_small  # noqa: E402

BF16 = torch.bfloat16


def _parts(cfg):
    """A parallel and a general layer of a configuration."""
    from tileinfer_b200.models.luvapel import GeneralDelta, ParallelMixer
    return tuple(next(L for L in cfg.layers if isinstance(L.mixer, k)) for k in (ParallelMixer, GeneralDelta))


def closest(cfg):
    """The hybrid-family configuration of the same size."""
    from tileinfer_b200.models.config import ModelConfig
    from tileinfer_b200.models.luvapel import ParallelMixer
    par, gen = _parts(cfg)
    a, g = par.mixer.left, gen.mixer
    return ModelConfig(name=f"hybrid-{cfg.hidden_size}", vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, num_layers=cfg.num_layers,
                       layer_types=tuple("full_attention" if isinstance(L.mixer, ParallelMixer) else "linear_attention" for L in cfg.layers),
                       intermediate_size=par.mlp.ff * 2 // 3, num_q_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, rotary_dim=a.rot_dims,
                       rope_theta=a.rot_base, gdn_num_k_heads=g.heads // 2, gdn_num_v_heads=g.heads, gdn_head_k_dim=g.dim, gdn_head_v_dim=g.dim,
                       max_position_embeddings=cfg.max_position_embeddings)


class Step:
    """A two-layer model (parallel, general) with the buffers of one step filled by running it once."""

    def __init__(self, cfg, lens, ctxs):
        from tileinfer_b200.models.delta_b200 import B200DeltaModel
        from tileinfer_b200.models.luvapel import make_weights
        from tileinfer_b200.models.reference_cpu import Batch
        small = replace(cfg, layers=_parts(cfg))
        m = self.m = B200DeltaModel(small, make_weights(small, "random:0", None, "cuda"), quant="bf16")
        per = max(ctxs) // 16 + 1
        m.alloc_cache(per * len(lens), 16, len(lens) + 1)
        for pages in m.cache.values():
            for t in pages:
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
        if max(lens) == 1:
            self.x.cu = None                                   # the form that a captured decode step has
        self.par, self.gen = m.layers
        self.left, self.right, self.general = small.layers[0].mixer.left, small.layers[0].mixer.right, small.layers[1].mixer

    def bufs(self, L):
        T, x = self.x.T, self.x
        return (x.proj[:T * L.n_proj].view(T, L.n_proj), x.left[:T * max(L.n_left, 1)].view(T, max(L.n_left, 1)), x.right[:T * L.n_right].view(T, L.n_right))


def kernels(cfg, prompt, ctx, batch):
    rows = kernel_rows(cfg, "prefill", [prompt], [prompt])
    torch.cuda.empty_cache()
    rows += kernel_rows(cfg, "decode", [1] * batch, [ctx] * batch)
    torch.cuda.empty_cache()
    return rows


def kernel_rows(cfg, tag, lens, ctxs):
    from tileinfer_b200.ops import functional as F
    F.L("base", "rows", "attention", "hybrid", "conv", "delta")
    s = Step(cfg, lens, ctxs)
    m, x, W, rows = s.m, s.x, cfg.hidden_size, []
    T, S, pre = x.T, len(lens), tag == "prefill"
    small = timed if pre else timed_small
    row = lambda name, us, **kw: rows.append(_row(f"{tag}: {name}", us, **kw))
    gemm = lambda n, k, out=2: {"flops": 2 * T * n * k, "nbytes": 2 * (n * k + T * k) + out * T * n}
    lin = lambda n, k: F.LinearW(torch.randn(n, k, device="cuda").to(BF16) * k ** -0.5, False, "cuda")
    rnd = lambda *z: torch.randn(*z, device="cuda").to(BF16)
    mc = closest(cfg)

    # ---- products
    kd, vd = mc.gdn_num_k_heads * 128, mc.gdn_num_v_heads * 128
    like = {"parallel": ((2 * mc.num_q_heads + 2 * mc.num_kv_heads) * mc.head_dim, mc.num_q_heads * mc.head_dim), "general": (2 * kd + 2 * vd + 2 * mc.gdn_num_v_heads, vd)}
    for name, L in (("parallel", s.par), ("general", s.gen)):
        proj, left, right = s.bufs(L)
        row(f"input product ({name})", timed(lambda: L.w_in(x.h, proj, F.GEPI_STORE, F.gemm_epilogue(bias=L.in_bias))), **gemm(L.n_proj, W), like="input product")
        if L.n_left:
            row("output product (attention)", timed(lambda: L.w_o(left, x.y, F.GEPI_STORE)), **gemm(W, L.n_left), like="output product")
        w = L.w_o2 if L.n_left else L.w_o
        row(f"output product ({name}, delta rule)", timed(lambda: w(right, x.y2, F.GEPI_STORE)), **gemm(W, L.n_right), like="output product")
        n, k = like[name]
        a, b, xa, ya, yb = lin(n, W), lin(W, k), rnd(T, k), torch.empty(T, n, dtype=BF16, device="cuda"), rnd(T, W)
        row(f"input product ({'attention' if name == 'parallel' else 'DeltaNet'}, other model)", timed(lambda: F.gemm_bf16(a, x.h, out=ya)), **gemm(n, W))
        row("output product (other model)", timed(lambda: F.gemm_bf16(b, xa, out=yb, epi=F.GEPI_ROWPAR, resid=yb)), **gemm(W, k, 4))
        del a, b, xa, ya
    L = s.par
    act = x.ff[:T * L.ff].view(T, L.ff)
    ex = F.gemm_epilogue(out2=act, n_split=W, bias=L.up_bias)
    row("up (squared) and gate logits", timed(lambda: L.w_up(x.h, x.gate, F.GEPI_SPLIT_RELU2, ex)), **gemm(L.ff + W, W), like="gate_up")
    row("down", timed(lambda: L.w_down(act, x.y, F.GEPI_STORE)), **gemm(W, L.ff), like="down")
    ff = mc.intermediate_size
    up, down, act2 = lin(2 * ff, W), lin(W, ff), rnd(T, ff)
    row("gate_up (other model)", timed(lambda: F.gemm_bf16(up, x.h, out=act2, epi=F.GEPI_SWIGLU)), flops=4 * T * W * ff, nbytes=2 * (2 * ff * W + T * (W + ff)))
    row("down (other model)", timed(lambda: F.gemm_bf16(down, act2, out=yb, epi=F.GEPI_ROWPAR, resid=yb)), **gemm(W, ff, 4))
    del up, down, act2
    # ---- the residual's row operations
    proj, left, right = s.bufs(s.par)
    gate, nw = proj[:, s.par.rg_col:], rnd(W)
    row("branch norms + gate + norm + residual", small(lambda: F.gated_norm(x.y, gate, x.x, L.norm1, x.h, W, 1e-6, y2=x.y2, w_y=L.left_out, w_y2=L.right_out, scale=0.5)),
        nbytes=16 * T * W, like="rmsnorm")
    row("gate + norm + residual", small(lambda: F.gated_norm(x.y, x.gate, x.x, L.norm2, x.h, W, 1e-6)), nbytes=14 * T * W, like="rmsnorm")
    row("norm + residual + next norm (Gerivik)", small(lambda: F.resid_norm(x.y, x.x, L.norm1, x.h, L.norm2, W, 1e-6)), nbytes=12 * T * W)
    row("rmsnorm (other model)", small(lambda: F.rmsnorm(yb, nw, 1e-6, out=x.h)), nbytes=4 * T * W)
    # ---- attention
    a = s.left
    H, G, D, win = a.heads, a.kv_heads, a.dim, a.window
    keys = sum(sum(min(p + 1, win) for p in range(c - n, c)) for n, c in zip(lens, ctxs))
    reach = sum(min(c, win + n - 1) for n, c in zip(lens, ctxs))
    prep = 2 * T * (2 * H + 3 * G) * D
    row("norms, rotation, store", small(lambda: m._rotate_and_store(s.par, x, proj)), nbytes=prep, like="qk norm")
    q, (kc, vc) = x.q[:T * H * D].view(T, H * D), m.cache[0]
    r, gq, zero, qq = F.QkvPrepParams(), rnd(T, (2 * H + 2 * G) * D), torch.zeros(D, dtype=BF16, device="cuda"), rnd(T, H * D)
    kc0, vc0 = torch.zeros_like(kc), torch.zeros_like(vc)
    r.proj, r.q_norm, r.k_norm, r.positions, r.slot_mapping, r.q_out, r.kcache, r.vcache = (
        t.data_ptr() for t in (gq, zero, zero, x.positions, x.slot_mapping, qq, kc0, vc0))
    r.ld, r.hq, r.hkv, r.rotary_dim, r.eps, r.log2_theta, r.num_blocks = gq.shape[1], H, G, a.rot_dims, 1e-6, math.log2(a.rot_base), m.num_blocks
    row("qk norm, rotation, store (other model)", small(lambda: F.qkv_prep(r, T, D)), nbytes=2 * T * (2 * H + 4 * G) * D)
    del kc0, vc0, qq
    cost = lambda k, n: {"flops": 4 * k * H * D, "nbytes": 2 * (T * 3 * H * D + 2 * n * G * D)}
    row("attention, window, gate", timed(lambda: m._attention(s.par, x, q, proj, left)), **cost(keys, reach), like="attention")
    whole = cost(sum(c * n - n * (n - 1) // 2 for n, c in zip(lens, ctxs)), sum(ctxs))
    if pre:
        row("attention over the context (other model)", timed(lambda: F.attn_prefill(q, kc, vc, m.num_blocks, x.block_tables, x.positions, x.tiles, gq, left, hq=H,
                                                                                     hkv=G, D=D, max_blocks=x.max_blocks, ld=gq.shape[1])), **whole)
    else:
        p = F.AttnParams()
        p.q, p.kcache, p.vcache, p.block_tables, p.positions = (t.data_ptr() for t in (q, kc, vc, x.block_tables, x.positions))
        p.qg_seq, p.qg_tok0, p.qg_ntok, p.o_part, p.ml_part, p.out = (t.data_ptr() for t in (*x.qg, x.o_part, x.ml_part, left))
        p.hq, p.hkv, p.rep, p.max_blocks, p.nsplit, p.num_qg, p.num_blocks = H, G, 1, x.max_blocks, x.nsplit, x.num_qg, m.num_blocks
        p.scale_log2e, p.gate_src, p.ld = a.scale * math.log2(math.e), gq.data_ptr(), gq.shape[1]
        row("attention over the context (other model)", timed(lambda: F.attn_paged(p, D, D)), **whole)
    del gq
    # ---- delta rules: algorithmic cost as for the like kernel (three products with the state per token; general: the same)
    for name, L, heads, kv, dk, dv in (("gated delta rule", s.par, s.right.heads, s.right.kv_heads, s.right.dim, s.right.vdim),
                                       ("general delta rule", s.gen, s.general.heads, s.general.heads, s.general.dim, s.general.dim)):
        proj, left, right = s.bufs(L)
        io = 2 * T * (2 * kv * dk + 3 * heads * dv + (2 * heads if L.n_left else heads * dk + L.R)) + 8 * S * heads * dk * dv
        state = {"flops": 6 * T * heads * dk * dv, "nbytes": io}
        row(f"{name}, all kernels", timed(lambda: m._delta(L, x, proj, right)), **state, like="gated DeltaNet")
        src = proj
        if L.n_left:
            row("  of it: convolutions", small(lambda: m._conv_inputs(L, x, proj)), nbytes=4 * T * L.C)
            src = m._conv_inputs(L, x, proj)
        p = m._delta_params(L, x, src, proj)
        if pre:
            ck, rng = x.chunks[F.delta_chunk_size(L.dk)]
            p.ck_seq, p.ck_tok0, p.ck_ntok, p.ck_snap = (z.data_ptr() for z in ck)
            p.long_seq, p.long_ck, p.nc, p.num_long = x.longs.data_ptr(), rng.data_ptr(), ck.shape[1], S
            p.t_ws, p.q_ws, p.s_ws, p.f_ws = (w.data_ptr() for w in m.delta_ws.get(p.nc, L.DH, L.dk, L.dv))
            row("  of it: chunk kernels", timed(lambda: F.delta_chunked(p, L.dk, L.dv, not L.parallel)), **state)
        else:
            row("  of it: state step", timed(lambda: F.delta_step(p, S, L.dk, L.dv, not L.parallel, False)), **state)
        o = x.o[:T * L.n_right].view(T, L.DH, L.dv)
        row("  of it: head norm + gate", small(lambda: F.head_norm(o, proj, L.dgate_col, L.h_norm, right, L.vdim, 1e-6, L.parallel)), nbytes=8 * T * heads * dv)
    rows.append(_like_gdn(F, tag, mc, T, S, pre))
    return rows


def run(args) -> dict:
    from tileinfer_b200.models.luvapel import LUVAPEL_2K, LUVAPEL_4K
    hbm, tf, basis = peaks()
    res = {"metric": "luvapel_tok_s", "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "higher_is_better": True,
           "dtype": "bf16", "data": "synthetic: random tokens, random weights", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "basis": basis},
           "sizes": {}}
    for cfg, prompt, ctx in ((LUVAPEL_2K, 8192, 2048), (LUVAPEL_4K, 8192, 4096)):
        rows = kernels(cfg, prompt, ctx, 64)
        ours = throughput(cfg, prompt, ctx, (1, 16, 64), args.steps, args.warmup)
        other = throughput(closest(cfg), prompt, ctx, (1, 16, 64), args.steps, args.warmup)
        res["sizes"][cfg.name] = {"layers": cfg.num_layers, "prompt": prompt, "context": ctx, "luvapel": ours, "hybrid_model": other, "kernels": rows}
        torch.cuda.empty_cache()
    res["value"] = res["sizes"]["luvapel-4k"]["luvapel"]["decode_64_tok_s"]
    res["config"] = {"model": "luvapel-4k", "global_batch": 64, "parallelism": "tp1", "cuda_graph": True,
                     "l2": "kernels: flushed between iterations; steps: more weights than L2"}
    return res


def table(res) -> str:
    lines = []
    for name, s in res["sizes"].items():
        lines.append(f"## {name}: {s['layers']} layers, prompt {s['prompt']}, decode context {s['context']}")
        keys = [k for k in s["luvapel"]]
        lines += [f"{k:20s} luvapel {s['luvapel'][k]:>12} other {s['hybrid_model'].get(k, '-'):>12}" for k in keys]
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
