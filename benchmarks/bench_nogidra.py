"""Nogidra beside the framework's closest model at equal size (`python bench.py --workload nogidra`).

The closest model is Gerivik: the same width, depth and vocabulary, gated linear attention with the same state bytes where
Nogidra has a parallel mixer, attention layers of the same head count and size elsewhere, and the same experts in every layer
(a dense layer of Nogidra is as wide as the experts a token uses together); bf16 weights.  Random weights.  Two parts:

  throughput  prefill of one prompt (eager step) and decode steps (captured graph) of 1, 16 and 64 sequences
  kernels     every kernel of Nogidra's layers and the like kernel of another model (Gerivik; Kabadra for latent attention, the
              hybrid model for plain attention and the recurrence), on the shapes of that step: time, algorithmic FLOPs or
              bytes, and the fraction of the measured peak

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
    """The latent, the parallel and the convolved layer of a configuration, and its experts."""
    from tileinfer_b200.models.nogidra import ConvAttention, ParallelMixer, RotaryLatent, SoftmaxExperts
    lay = [next(L for L in cfg.layers if isinstance(L.mixer, k)) for k in (RotaryLatent, ParallelMixer, ConvAttention)]
    return (*lay, next(L.mlp for L in cfg.layers if isinstance(L.mlp, SoftmaxExperts)))


def closest(cfg):
    """The Gerivik configuration of the same size."""
    from tileinfer_b200.models.gerivik import CappedAttention, GatedLinearAttention, GerivikConfig, GerivikLayer, RoutedExperts
    from tileinfer_b200.models.nogidra import ParallelMixer
    _, par, conv, f = _parts(cfg)
    mlp = RoutedExperts(experts=f.experts, identity=0, top=f.top, groups=8, keep=4, ff=f.ff, limit=7.0)
    a, r = conv.mixer, par.mixer.right
    attn = GerivikLayer(CappedAttention(heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, rot_base=5e5, rot_dims=a.dim // 4, scale=a.scale, softcap=40.0), mlp)
    gla = GerivikLayer(GatedLinearAttention(heads=r.inner * r.state // (128 * 256), dim=128, vdim=256, tau=12.0), mlp)
    return GerivikConfig(name=f"gerivik-{cfg.hidden_size}", vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, rms_eps=1e-6, embedding_scale=1.0,
                         max_position_embeddings=cfg.max_position_embeddings,
                         layers=tuple(gla if isinstance(L.mixer, ParallelMixer) else attn for L in cfg.layers))


class Step:
    """A three-layer model (latent, parallel, attention; dense, experts, dense) with the buffers of one step filled by running
    it once."""

    def __init__(self, cfg, lens, ctxs):
        from tileinfer_b200.models.mixed_b200 import B200MixedModel
        from tileinfer_b200.models.nogidra import DenseGlu, make_weights
        from tileinfer_b200.models.reference_cpu import Batch
        lat, par, conv, f = _parts(cfg)
        dense = next(L.mlp for L in cfg.layers if isinstance(L.mlp, DenseGlu))
        small = replace(cfg, layers=(replace(lat, mlp=dense), replace(par, mlp=f), replace(conv, mlp=dense)))
        m = self.m = B200MixedModel(small, make_weights(small, "random:0", None, "cuda"), quant="bf16")
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
        self.lat, self.par, self.conv = m.layers
        self.layers = small.layers

    def bufs(self, L):
        T, x = self.x.T, self.x
        return x.proj[:T * L.n_proj].view(T, L.n_proj), x.mix[:T * L.n_mix].view(T, L.n_mix)


def kernels(cfg, prompt, ctx, batch):
    rows = kernel_rows(cfg, "prefill", [prompt], [prompt])
    torch.cuda.empty_cache()
    rows += kernel_rows(cfg, "decode", [1] * batch, [ctx] * batch)
    torch.cuda.empty_cache()
    return rows


def kernel_rows(cfg, tag, lens, ctxs):
    from tileinfer_b200.ops import functional as F
    F.L("base", "rows", "attention", "hybrid", "latent", "conv", "ssd", "moe")
    s = Step(cfg, lens, ctxs)
    m, x, W, rows = s.m, s.x, cfg.hidden_size, []
    T, S, pre, ctx = x.T, len(lens), tag == "prefill", max(ctxs)
    small = timed if pre else timed_small
    row = lambda name, us, **kw: rows.append(_row(f"{tag}: {name}", us, **kw))
    gemm = lambda n, k, out=2: {"flops": 2 * T * n * k, "nbytes": 2 * (n * k + T * k) + out * T * n}
    lin = lambda n, k: F.LinearW(torch.randn(n, k, device="cuda").to(BF16) * k ** -0.5, False, "cuda")
    rnd = lambda *z: torch.randn(*z, device="cuda").to(BF16)
    pairs = lambda win: sum(sum(min(p + 1, win) for p in range(c - n, c)) for n, c in zip(lens, ctxs))
    reach = lambda win: sum(min(c, win + n - 1) for n, c in zip(lens, ctxs))
    silu = (math.inf, 1.0, 0.0)

    # ---- products
    for name, L in (("latent", s.lat), ("parallel", s.par), ("attention", s.conv)):
        proj, mix = s.bufs(L)
        ex = None if L.in_bias is None else F.gemm_epilogue(bias=L.in_bias)
        row(f"input product ({name}{', biases' if ex else ''})", timed(lambda: L.w_in(x.h, proj, F.GEPI_STORE, ex)), **gemm(L.n_proj, W), like="product")
        row(f"output product ({name}, into the fp32 residual)", timed(lambda: L.w_o(mix, x.x, F.GEPI_RESID32, F.gemm_epilogue(resid32=x.x))), **gemm(W, L.n_mix, 8), like="product")
    n, k = s.conv.n_proj, s.conv.n_mix
    a, b, ya, yb, xb = lin(n, W), lin(W, k), rnd(T, n), rnd(T, W), rnd(T, k)
    row("input product (other model)", timed(lambda: F.gemm_bf16(a, x.h, out=ya)), **gemm(n, W))
    row("output product (other model)", timed(lambda: F.gemm_bf16(b, xb, out=yb)), **gemm(W, k))
    del a, b, ya, xb
    L = s.lat
    act = x.ff[:T * L.ff].view(T, L.ff)
    row("gate/up + gated unit, biases", timed(lambda: L.w_up(x.h, act, F.GEPI_SPLIT_GLU, F.gemm_epilogue(out2=act, n_split=0, glu=silu, bias=L.up_bias))),
        flops=4 * T * W * L.ff, nbytes=2 * (2 * L.ff * W + T * (W + L.ff)), like="gate_up")
    row("down, bias, into the fp32 residual", timed(lambda: L.w_down(act, x.x, F.GEPI_RESID32, F.gemm_epilogue(resid32=x.x, bias=L.down_bias))), **gemm(W, L.ff, 8), like="down")
    up, down = lin(2 * L.ff, W), lin(W, L.ff)
    row("gate_up (other model)", timed(lambda: F.gemm_bf16(up, x.h, out=act, epi=F.GEPI_SWIGLU)), flops=4 * T * W * L.ff, nbytes=2 * (2 * L.ff * W + T * (W + L.ff)))
    row("down (other model)", timed(lambda: F.gemm_bf16(down, act, out=yb, epi=F.GEPI_ROWPAR, resid=yb)), **gemm(W, L.ff, 4))
    del up, down
    # ---- norms, routing, experts
    nw = rnd(W)
    row("norm of the fp32 residual", small(lambda: F.rmsnorm_f32(x.x, s.lat.norm1, x.h, W, 1e-6)), nbytes=6 * T * W, like="rmsnorm")
    row("rmsnorm (other model)", small(lambda: F.rmsnorm(yb, nw, 1e-6, out=x.h)), nbytes=4 * T * W)
    L, f = s.par, s.par.moe
    g = x.groups[(f.experts, f.choices, f.top)]
    xs, act = x.xs[:g.rows * m.Wp].view(g.rows, m.Wp), x.act[:g.rows * L.ff].view(g.rows, L.ff)
    corr, wn, y = torch.zeros(f.experts, device="cuda"), torch.ones(m.Wp, device="cuda"), rnd(T, m.Wp)
    if g.row_stride:
        row("norm + router + routing + rows to experts", small(lambda: m._norm_and_route(L, x, None, None)), nbytes=6 * W * T + 2 * W * (f.experts + T * f.top), like="norm + routing")
        row("norms + residual + router + routing + rows to experts (other model)",
            small(lambda: F.moe_norm_route(y, x.x, wn, x.h, L.norm2, W, 1e-6, g, L.router_rows, corr, 8, 4, xs)), nbytes=12 * W * T + 2 * W * (f.experts + T * f.top))
    else:
        lg = x.logits[:T * f.experts].view(T, f.experts)
        row("router product", small(lambda: L.router(x.h, lg, F.GEPI_F32)), **gemm(f.experts, W, 4))
        row("routing", small(lambda: F.moe_route(g, lg, None, 1, 1)), nbytes=T * (4 * f.experts + 12 * f.top), like="routing")
        row("routing (other model)", small(lambda: F.moe_route(g, lg, corr, 8, 4)), nbytes=T * (4 * f.experts + 12 * f.top))
        row("token rows to experts", small(lambda: F.moe_permute(g, x.h, xs)), nbytes=2 * W * T * (1 + f.top), like="rmsnorm")
    live, used = int((g.ids >= 0).sum()), int(torch.unique(g.ids[g.ids >= 0]).numel())
    ex = F.gemm_epilogue(out2=act, n_split=0, glu=silu)
    row(f"experts gate/up + gated unit ({used} experts, {live} rows)", timed(lambda: L.w_up(xs, g, None, F.GEPI_SPLIT_GLU, ex)), flops=4 * live * W * L.ff,
        nbytes=2 * (used * 2 * L.ff * W + live * (W + L.ff)), like="gate_up")
    ye = torch.empty_like(xs)
    row("experts down", timed(lambda: L.w_down(act, g, ye, F.GEPI_STORE)), flops=2 * live * W * L.ff, nbytes=2 * (used * L.ff * W + live * (W + L.ff)), like="down")
    row("experts' sum + residual + next norm", small(lambda: F.resid_norm(ye, x.x, None, x.h, L.norm1, W, 1e-6, routed=g)), nbytes=2 * W * (live + T) + 8 * W * T, like="experts' sum")
    row("experts' sum + norm + residual + next norm (other model)", small(lambda: F.resid_norm(ye, x.x, wn, x.h, L.norm1, W, 1e-6, routed=g)), nbytes=2 * W * (live + T) + 8 * W * T)
    del ye, y
    rows += _latent_rows(F, s, tag, small, pairs, reach, S)
    rows += _attention_rows(F, s, tag, small, pairs, reach, ctx)
    # ---- state-space mixer
    L, r = s.par, s.layers[1].mixer.right
    proj, mix = s.bufs(L)
    io = 2 * T * (3 * r.inner + 2 * r.groups * r.state) + 8 * S * r.inner * r.state
    row("state-space mixer, all kernels", timed(lambda: m._state_space(L, x, proj, mix)), flops=4 * T * r.inner * r.state, nbytes=io, like="recurrence")
    row("  of it: convolution", small(lambda: m._conv_inputs(L, x, proj)), nbytes=4 * T * r.conv_channels)
    p = m._ssd_params(L, x, x.xbc[:T * L.C].view(T, L.C), proj, mix)
    run = (lambda: F.ssd_chunked(p, L.Np)) if pre else (lambda: F.ssd_step(p, S, L.Np, False))
    row("  of it: chunk kernels" if pre else "  of it: state step", timed(run), flops=4 * T * r.inner * r.state,
        nbytes=2 * T * (r.inner + 2 * r.groups * r.state) + 4 * T * r.inner + 8 * S * r.inner * r.state, like="recurrence")
    row("  of it: gate + group norm", small(lambda: F.ssd_finish(p, T, False)), nbytes=8 * T * r.inner, like="rmsnorm")
    from benchmarks.bench_gerivik import closest as hybrid
    rows.append(_like_gdn(F, tag, hybrid(closest(cfg)), T, S, pre))
    return rows


def _latent_rows(F, s, tag, small, pairs, reach, S):
    """Latent attention with a rotated part, beside Kabadra's."""
    m, x, L, rows = s.m, s.x, s.lat, []
    row = lambda name, us, **kw: rows.append(_row(f"{tag}: {name}", us, **kw))
    proj, mix = s.bufs(L)
    T, H, R, P, win, D, V = x.T, L.heads, L.R, s.layers[0].mixer.rot_dim, L.window, L.dim, s.layers[0].mixer.vdim
    cache = m._latent_rows(L)
    row("rotation, latent norm, store", small(lambda: F.latent_rope(proj, H, L.dp, D, L.kv_col, L.kv_norm, L.inv_freq, x.positions, x.slot_mapping, cache, R, 1e-6)),
        nbytes=2 * T * (2 * H * P + 2 * (R + P)), like="latent store")
    other = torch.zeros(cache.shape[0], 16, L.Ro, dtype=BF16, device="cuda")
    row("latent norm, store (other model)", small(lambda: F.latent_store(proj, L.kv_col, L.kv_norm, x.slot_mapping, other, R, 1e-6)), nbytes=4 * T * R)
    if tag == "prefill":
        slots, tiles = x.reach[win]
        n = slots.numel()
        lat = x.latents[(cache.data_ptr(), win)]
        kv = torch.empty(n, L.w_ukv.N, dtype=BF16, device="cuda")
        row("rows in reach", small(lambda: F.latent_gather(cache, slots, lat)), nbytes=4 * n * L.Rp)
        row("keys and values from latents", timed(lambda: F.gemm_bf16(L.w_ukv, lat, out=kv)), flops=2 * n * L.w_ukv.N * L.Rp,
            nbytes=2 * n * (L.Rp + L.w_ukv.N) + 2 * L.w_ukv.N * L.Rp, like="keys and values")
        w0 = F.LinearW(torch.randn(H * (D + V), R, device="cuda").to(BF16), False, "cuda")
        l0, kv0 = lat[:, :R].contiguous(), torch.empty(n, H * (D + V), dtype=BF16, device="cuda")
        row("keys and values from latents (other model)", timed(lambda: F.gemm_bf16(w0, l0, out=kv0)), flops=2 * n * w0.N * R, nbytes=2 * n * (R + w0.N) + 2 * w0.N * R)
        row(f"attention, window {win}", timed(lambda: F.latent_prefill(proj, kv, tiles, mix, H=H, dp=L.dp, vp=L.vp, window=win, scale=L.scale)),
            flops=2 * pairs(win) * H * (D + P + V), like="latent attention")
        q0, gate = torch.randn(T, H * D + H, device="cuda").to(BF16), torch.zeros(H, device="cuda")
        row("attention (other model)", timed(lambda: F.latent_prefill(q0, kv0, tiles, mix, H=H, dp=D, vp=V, window=win, scale=L.scale, sink=gate, gate=q0, gcol=H * D)),
            flops=2 * pairs(win) * H * (D + V))
        return rows
    q, o = x.q_abs[:T * H * L.Rp].view(T, H * L.Rp), x.o_lat[:T * H * L.Ro].view(T, H * L.Ro)
    row("W_uk into the query", small(lambda: F.head_product(proj, L.uk_t, q)), flops=2 * T * H * D * R, nbytes=2 * H * D * R + 2 * T * H * (D + 2 * P + R), like="head product")
    uk0, x0, q0 = (torch.randn(*z, device="cuda").to(BF16) for z in ((H, R, D), (T, H * D), (T, H * R)))
    row("W_uk into the query (other model)", small(lambda: F.head_product(x0, uk0, q0)), flops=2 * T * H * D * R, nbytes=2 * H * D * R + 2 * T * H * (D + R))
    p = F.LatentAttnParams()
    ns = m._latent_nsplit(L, S)
    p.nsplit, p.q, p.out = ns, q.data_ptr(), o.data_ptr()
    p.cache, p.block_tables, p.positions = cache.data_ptr(), x.block_tables.data_ptr(), x.positions.data_ptr()
    p.qg_seq, p.qg_tok0, p.qg_ntok = (t.data_ptr() for t in x.qg)
    if ns > 1:
        p.o_part, p.ml_part = x.lat_part.data_ptr(), x.lat_ml.data_ptr()
    p.H, p.R, p.Rp, p.Ro, p.max_blocks, p.num_qg, p.window, p.num_blocks, p.scale = H, R, L.Rp, L.Ro, x.max_blocks, S, win, m.num_blocks, L.scale
    keys = reach(win)
    row("attention over latents", timed(lambda: F.latent_attn(p, False)), flops=2 * keys * H * (2 * R + P), nbytes=2 * keys * (R + P) + 2 * T * H * (2 * R + P), like="latent attention")
    p.cache, p.q, p.Rp, p.Ro = other.data_ptr(), q0.data_ptr(), L.Ro, L.Ro
    row("attention over latents (other model)", timed(lambda: F.latent_attn(p, False)), flops=4 * keys * H * R, nbytes=2 * keys * R + 4 * T * H * R)
    row("W_uv", small(lambda: F.head_product(o, L.uv, mix)), flops=2 * T * H * V * R, nbytes=2 * H * V * R + 2 * T * H * (V + R), like="head product")
    return rows


def _attention_rows(F, s, tag, small, pairs, reach, ctx):
    """Convolved and normed heads, windowed paged attention, beside rotated heads and plain attention."""
    m, x, rows = s.m, s.x, []
    T, S, pre = x.T, x.S, tag == "prefill"
    row = lambda name, us, **kw: rows.append(_row(f"{tag}: {name}", us, **kw))
    for name, L, prep, spec in (("convolutions, temperature, store", s.conv, m._conv_heads, s.layers[2].mixer),
                                ("norms, rotation, store", s.par, m._normed_heads, s.layers[1].mixer.left)):
        proj, mix = s.bufs(L)
        H, G, D, win = spec.heads, spec.kv_heads, spec.dim, spec.window
        row(name, small(lambda: prep(L, x, proj)), nbytes=4 * T * (H + 2 * G) * D, like="heads and store")
        q = prep(L, x, proj)
        row(f"attention, window {win}" + (", slopes, gate" if L.slopes is not None else ""), timed(lambda: m._attention(L, x, q, proj, mix)),
            flops=4 * pairs(win) * H * D, nbytes=2 * (2 * T * H * D + 2 * reach(win) * G * D), like="attention")
    H, G, D = spec.heads, spec.kv_heads, spec.dim
    kc, vc = (torch.zeros_like(t) for t in m.cache[1])
    proj, q = torch.randn(T, (H + 2 * G) * D, device="cuda").to(BF16), torch.zeros(T, H * D, dtype=BF16, device="cuda")
    inv = torch.ones(D // 8, device="cuda")
    r = F.RopeUnitParams()
    r.proj, r.inv_freq, r.positions, r.slot_mapping, r.q_out, r.kcache, r.vcache = (t.data_ptr() for t in (proj, inv, x.positions, x.slot_mapping, q, kc, vc))
    r.T, r.ld, r.k_col, r.v_col, r.H, r.G, r.dim, r.dp, r.vp, r.half, r.num_blocks, r.eps = T, proj.shape[1], H * D, (H + G) * D, H, G, D, D, D, D // 8, m.num_blocks, 1e-6
    row("rotated unit heads, store (other model)", small(lambda: F.rope_unit(r, False)), nbytes=4 * T * (H + 2 * G) * D)
    kc.normal_(), vc.normal_()
    keys = sum([c * (c + 1) // 2 for c in [ctx]]) if pre else S * ctx
    out = torch.zeros(T, H * D, dtype=BF16, device="cuda")
    if pre:
        run = lambda: F.attn_prefill(q, kc, vc, m.num_blocks, x.block_tables, x.positions, x.tiles, None, out, hq=H, hkv=G, D=D, max_blocks=x.max_blocks, ld=0)
    else:
        a = F.AttnParams()
        a.q, a.kcache, a.vcache, a.block_tables, a.positions, a.out = (t.data_ptr() for t in (q, kc, vc, x.block_tables, x.positions, out))
        a.qg_seq, a.qg_tok0, a.qg_ntok, a.o_part, a.ml_part = (t.data_ptr() for t in (*x.qg, x.o_part, x.ml_part))
        a.hq, a.hkv, a.rep, a.max_blocks, a.nsplit, a.num_qg, a.num_blocks, a.scale_log2e = H, G, 1, x.max_blocks, x.nsplit, S, m.num_blocks, 0.1
        run = lambda: F.attn_paged(a, D)
    row(f"attention over {ctx} keys (other model)", timed(run), flops=4 * keys * H * D, nbytes=2 * (2 * T * H * D + 2 * S * ctx * G * D))
    return rows


def run(args) -> dict:
    from tileinfer_b200.models.nogidra import NOGIDRA_2K, NOGIDRA_4K
    hbm, tf, basis = peaks()
    res = {"metric": "nogidra_tok_s", "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "higher_is_better": True,
           "dtype": "bf16", "data": "synthetic: random tokens, random weights", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "basis": basis},
           "sizes": {}}
    for cfg, prompt, ctx in ((NOGIDRA_2K, 8192, 2048), (NOGIDRA_4K, 8192, 4096)):
        rows = kernels(cfg, prompt, ctx, 64)
        ours = throughput(cfg, prompt, ctx, (1, 16, 64), args.steps, args.warmup)
        other = throughput(closest(cfg), prompt, ctx, (1, 16, 64), args.steps, args.warmup)
        res["sizes"][cfg.name] = {"layers": cfg.num_layers, "prompt": prompt, "context": ctx, "nogidra": ours, "gerivik_model": other, "kernels": rows}
        torch.cuda.empty_cache()
    res["value"] = res["sizes"]["nogidra-4k"]["nogidra"]["decode_64_tok_s"]
    res["config"] = {"model": "nogidra-4k", "global_batch": 64, "parallelism": "tp1", "cuda_graph": True,
                     "l2": "kernels: flushed between iterations; steps: more weights than L2"}
    return res


def table(res) -> str:
    lines = []
    for name, s in res["sizes"].items():
        lines.append(f"## {name}: {s['layers']} layers, prompt {s['prompt']}, decode context {s['context']}")
        lines += [f"{k:20s} nogidra {s['nogidra'][k]:>12} other {s['gerivik_model'].get(k, '-'):>12}" for k in s["nogidra"]]
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
