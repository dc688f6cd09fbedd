"""Kabadra beside the framework's closest model at equal size (`python bench.py --workload kabadra`).

The closest model is the hybrid family with attention layers only: same width, depth, head count and size, feed-forward
and vocabulary, bf16 weights, KV heads = heads / 4, full causal attention.  Random weights.  Two parts:

  throughput  prefill of one prompt (eager step) and decode steps (captured graph) of 1, 16 and 64 sequences
  kernels     every kernel of a Kabadra layer and the like kernel of the other model, alone, on the shapes of that step:
              time, algorithmic FLOPs or bytes, and the fraction of the measured peak

CUDA events on the launching stream after warm-up.  Between timed iterations the L2 is flushed (kernels) or the step
streams more weights than it holds (throughput).
"""
from __future__ import annotations

import json
import math
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

BF16 = torch.bfloat16


def peaks():
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return d["hbm_gbs"], d["bf16_tflops"], "of measured"
    except Exception:
        return 6650.0, 1590.0, "of fallback"


def closest(cfg):
    """The hybrid-family configuration of the same size, attention layers only."""
    from tileinfer_b200.models.config import ModelConfig
    m, f = cfg.layers[0].mixer, cfg.layers[0].mlp
    n = cfg.num_layers
    return ModelConfig(name=f"attention-{cfg.hidden_size}", vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size, num_layers=n,
                       layer_types=("full_attention",) * n, intermediate_size=f.ff, num_q_heads=m.heads,
                       num_kv_heads=max(1, m.heads // 4), head_dim=m.dim, rotary_dim=m.dim // 4, rope_theta=1e6,
                       gdn_num_k_heads=1, gdn_num_v_heads=1, gdn_head_k_dim=64, gdn_head_v_dim=64,
                       max_position_embeddings=cfg.max_position_embeddings)


_FLUSH = None


def timed_small(fn, repeat=20):
    """Microseconds of one fn() of `repeat` in a captured graph: for kernels of a few microseconds, which a pair of events
    around one launch would not resolve.  Their inputs stay in the L2, as they do inside a step."""
    fn()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for _ in range(repeat):
            fn()
    return timed(g.replay, flush=False) / repeat


def timed(fn, n=12, warm=3, flush=True):
    """Median microseconds of fn() between two events."""
    global _FLUSH
    if flush and _FLUSH is None:
        _FLUSH = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
    for _ in range(warm):
        fn()
    ts = []
    for _ in range(n):
        if flush:
            _FLUSH.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b) * 1e3)
    return sorted(ts)[len(ts) // 2]


# ---------------------------------------------------------------------------------------------------- throughput
def throughput(mc, prompt, ctx, batches, steps, warmup):
    """Tokens per second of one model: {"prefill": ..., "decode_<n>": ...}."""
    import gc
    from tileinfer_b200.engine.config import Config
    from tileinfer_b200.engine.model_runner import ModelRunner
    from tileinfer_b200.models.reference_cpu import Batch
    from tileinfer_b200.parallel.comm import init_distributed
    top = max(batches)
    cfg = Config("bench", model_config=mc, quantization="bf16", device="cuda", max_num_seqs=top, max_model_len=max(prompt, ctx) + 64,
                 num_kvcache_blocks=max(top * (ctx // 16 + 2), prompt // 16 + 2), enable_prefix_caching=False)
    r = ModelRunner(cfg, init_distributed(1, 60, "cuda"))
    model = r.load_model()
    r.allocate_kv_cache()
    model.capture_decode_graphs(1, 1, cfg.max_model_len, r.padding_deltanet_slot)
    out = {"weights_gb": round(model.weight_bytes() / 1e9, 2)}
    g = torch.Generator().manual_seed(1)
    table = list(range(prompt // 16 + 1))
    b = Batch(torch.randint(0, mc.vocab_size, (prompt,), generator=g), torch.arange(prompt), [0, prompt], [prompt], [table],
              torch.arange(prompt), [0])
    us = timed(lambda: model.logits(model.forward(b)), n=max(3, steps // 4), warm=warmup, flush=False)
    out["prefill_tok_s"], out["prefill_ms"] = round(prompt / us * 1e6), round(us / 1e3, 3)
    for n in batches:
        model.buckets = [n]
        gr = model._get_graph(n, 1, model.fused_argmax_ok(n, 1))
        per = ctx // 16 + 1
        tables = [list(range(i * per, (i + 1) * per)) for i in range(n)]
        p = ctx - 1
        model._decode_graph_step(Batch(torch.randint(0, mc.vocab_size, (n,), generator=g), torch.full((n,), p), list(range(n + 1)), [p + 1] * n,
                                       tables, torch.tensor([t[p // 16] * 16 + p % 16 for t in tables]), list(range(n))), 1)
        us = timed(gr.graph.replay, n=steps, warm=warmup, flush=False)
        out[f"decode_{n}_tok_s"], out[f"decode_{n}_ms"] = round(n / us * 1e6, 1), round(us / 1e3, 4)
        out["launches_per_step"] = gr.launches
    model.release_graphs()
    del r, model, gr
    gc.collect()
    torch.cuda.empty_cache()
    return out


# ---------------------------------------------------------------------------------------------------- kernels
def _row(name, us, *, flops=0, nbytes=0, like=None):
    hbm, tf, _ = peaks()
    floor = max(flops / (tf * 1e6), nbytes / (hbm * 1e3))
    return {"kernel": name, "us": round(us, 2), "floor_us": round(floor, 2), "fraction": round(floor / us, 3),
            "bound": "tensor" if flops / (tf * 1e6) > nbytes / (hbm * 1e3) else "memory", "like": like}


def kernels(cfg, prompt, ctx, batch):
    """Rows of the kernel table for one size: a prefill step of `prompt` tokens and a decode step of `batch` sequences."""
    from tileinfer_b200.ops import functional as F
    F.L("base", "rows", "attention", "hybrid", "latent")
    m, f = cfg.layers[0].mixer, cfg.layers[0].mlp
    W, H, D, R, ff, win = cfg.hidden_size, m.heads, m.dim, m.kv_rank, f.ff, m.window
    dev, rows = "cuda", []
    rnd = lambda *s: torch.randn(*s, device=dev).to(BF16)
    lin = lambda n, k: F.LinearW(torch.randn(n, k, device=dev).to(BF16) * k ** -0.5, False, dev)
    sink, norm_w, norm_r = torch.zeros(H, device=dev), torch.ones(W, device=dev), torch.ones(R, device=dev)
    n_proj = H * D + R + -(-H // 8) * 8
    w_in, w_out, w_ukv = lin(n_proj + 2 * ff, W), lin(W, H * m.vdim + ff), lin(H * (D + m.vdim), R)
    like_up, like_down = lin(2 * ff, W), lin(W, ff)
    for T, tag in ((prompt, "prefill"), (batch, "decode")):
        x, h, proj, cat = torch.randn(T, W, device=dev), rnd(T, W), rnd(T, n_proj), rnd(T, H * m.vdim + ff)
        ex = F.gemm_epilogue(out2=cat[:, H * m.vdim:], n_split=n_proj, glu=(f.limit, 1.702, 1.0))
        rows.append(_row(f"{tag}: input product + gated unit", timed(lambda: F.gemm_bf16(w_in, h, out=proj, epi=F.GEPI_SPLIT_GLU, ex=ex)),
                         flops=2 * T * W * w_in.N, nbytes=2 * (w_in.N * W + T * (W + n_proj + ff)), like="gate_up"))
        act = rnd(T, ff)
        rows.append(_row(f"{tag}: gate_up (other model)", timed(lambda: F.gemm_bf16(like_up, h, out=act, epi=F.GEPI_SWIGLU)),
                         flops=2 * T * W * 2 * ff, nbytes=2 * (2 * ff * W + T * (W + ff))))
        rows.append(_row(f"{tag}: output product + fp32 residual",
                         timed(lambda: F.gemm_bf16(w_out, cat, out=x, epi=F.GEPI_RESID32, ex=F.gemm_epilogue(resid32=x))),
                         flops=2 * T * W * w_out.K, nbytes=2 * (w_out.K * W + T * w_out.K) + 8 * T * W, like="down"))
        hb = rnd(T, W)
        rows.append(_row(f"{tag}: down (other model)", timed(lambda: F.gemm_bf16(like_down, act, out=hb, epi=F.GEPI_ROWPAR, resid=hb)),
                         flops=2 * T * W * ff, nbytes=2 * (ff * W + T * ff) + 4 * T * W))
        rows.append(_row(f"{tag}: RMSNorm of the fp32 residual", (timed if tag == "prefill" else timed_small)(lambda: F.rmsnorm_f32(x, norm_w, h, W, 1e-6)), nbytes=6 * T * W,
                         like="rmsnorm"))
        nw = rnd(W)
        rows.append(_row(f"{tag}: rmsnorm (other model)", (timed if tag == "prefill" else timed_small)(lambda: F.rmsnorm(hb, nw, 1e-6, out=h)), nbytes=4 * T * W))
        cache = torch.zeros(T // 16 + 1, 16, R, dtype=BF16, device=dev)
        slots = torch.arange(T, device=dev)
        rows.append(_row(f"{tag}: latent norm + store", timed_small(lambda: F.latent_store(proj, H * D, norm_r, slots, cache, R, 1e-6)),
                         nbytes=4 * T * R))
        del x, h, proj, cat, act, hb, cache
    # ---- prefill attention: one sequence, whole prompt
    T = prompt
    proj, out = rnd(T, n_proj), torch.empty(T, H * m.vdim, dtype=BF16, device=dev)
    lat, kv = rnd(T, R), torch.empty(T, w_ukv.N, dtype=BF16, device=dev)
    rows.append(_row("prefill: keys and values from latents", timed(lambda: F.gemm_bf16(w_ukv, lat, out=kv)), flops=2 * T * R * w_ukv.N,
                     nbytes=2 * (T * R + T * w_ukv.N + R * w_ukv.N), like="gate_up"))
    kv.normal_()
    tiles = sorted([(a, min(128, T - a), a, 0, 0) for a in range(0, T, 128)], key=lambda t: -min(t[2] + t[1], win))
    tiles = torch.tensor(tiles, dtype=torch.int32).t().contiguous().to(dev)
    pairs = sum(min(i + 1, win) for i in range(T))
    us = timed(lambda: F.latent_prefill(proj, kv, tiles, out, H=H, dp=D, vp=m.vdim, window=win, scale=m.scale, sink=sink, gate=proj, gcol=H * D + R))
    rows.append(_row(f"prefill: attention, window {win}", us, flops=2 * pairs * H * (D + m.vdim), like="attention prefill"))
    hkv, nb = max(1, H // 4), T // 16
    q, kc = rnd(T, H * D), rnd(nb, hkv * 16 * D)
    vc, bt = rnd(nb, hkv * 16 * D), torch.arange(nb, dtype=torch.int32, device=dev)[None].contiguous()
    pos, ld = torch.arange(T, dtype=torch.int32, device=dev), H * 2 * D
    gate, t3 = rnd(T, ld), torch.stack([torch.zeros_like(tiles[0]), tiles[0], tiles[1]]).contiguous()
    t3 = t3[:, torch.argsort(t3[1], descending=True)].contiguous()
    us = timed(lambda: F.attn_prefill(q, kc, vc, nb, bt, pos, t3, gate, out, hq=H, hkv=hkv, D=D, max_blocks=nb, ld=ld))
    rows.append(_row("prefill: full attention (other model)", us, flops=2 * (T * (T + 1) // 2) * H * 2 * D))
    del proj, out, lat, kv, q, kc, vc, gate
    rows += decode_attention(F, cfg, ctx, batch)
    return rows


def decode_attention(F, cfg, ctx, S):
    m, dev, rows = cfg.layers[0].mixer, "cuda", []
    H, D, R, win = m.heads, m.dim, m.kv_rank, m.window
    rnd = lambda *s: torch.randn(*s, device=dev).to(BF16)
    nb = ctx // 16
    idx, one = torch.arange(S, dtype=torch.int32, device=dev), torch.ones(S, dtype=torch.int32, device=dev)
    bt, pos = torch.arange(S * nb, dtype=torch.int32, device=dev).view(S, nb), torch.full((S,), ctx - 1, dtype=torch.int32, device=dev)
    x, uk, uv, q, gate = rnd(S, H * D), rnd(H, R, D), rnd(H, m.vdim, R), rnd(S, H * R), rnd(S, H * D + H)
    rows.append(_row("decode: W_uk into the query", timed_small(lambda: F.head_product(x, uk, q)), flops=2 * S * H * R * D, nbytes=2 * (H * R * D + S * H * (R + D))))
    o, out = rnd(S, H * R), torch.empty(S, H * m.vdim, dtype=BF16, device=dev)
    rows.append(_row("decode: W_uv and the gate", timed_small(lambda: F.head_product(o, uv, out, gate=gate, gcol=H * D)), flops=2 * S * H * R * m.vdim,
                     nbytes=2 * (H * R * m.vdim + S * H * (R + m.vdim))))
    cache, sink = rnd(S * nb, 16, R), torch.zeros(H, device=dev)
    p = F.LatentAttnParams()
    p.nsplit = F.latent_nsplit(S, H, R, win)
    part = torch.empty(F.latent_part_floats(S, H, R, p.nsplit), device=dev)
    ml = torch.empty(part.numel() // 32 + 64, device=dev)
    p.q, p.cache, p.out, p.sink = q.data_ptr(), cache.data_ptr(), o.data_ptr(), sink.data_ptr()
    p.block_tables, p.positions, p.qg_seq, p.qg_tok0, p.qg_ntok = bt.data_ptr(), pos.data_ptr(), idx.data_ptr(), idx.data_ptr(), one.data_ptr()
    p.o_part, p.ml_part = part.data_ptr(), ml.data_ptr()
    p.H, p.R, p.Rp, p.max_blocks, p.num_qg, p.window, p.num_blocks, p.scale = H, R, R, nb, S, win, S * nb, m.scale
    keys = min(ctx, win)
    rows.append(_row(f"decode: attention over {keys} latents, {S} sequences", timed(lambda: F.latent_attn(p, False)), flops=4 * S * H * keys * R,
                     nbytes=2 * S * (keys * R + 2 * H * R), like="attention decode"))
    del cache, part
    hkv = max(1, H // 4)
    G = H // hkv
    kc, vc, ld = rnd(S * nb, hkv * 16 * D), rnd(S * nb, hkv * 16 * D), H * 2 * D
    qq, gg = rnd(S, H * D), rnd(S, ld)
    a = F.AttnParams()
    ns = max(1, min(32, -(-8 * F.NUM_SMS // (S * hkv))))
    op, mp = torch.empty(S * hkv * ns * 16 * D, device=dev), torch.empty(S * hkv * ns * 32, device=dev)
    a.q, a.kcache, a.vcache, a.block_tables, a.positions = qq.data_ptr(), kc.data_ptr(), vc.data_ptr(), bt.data_ptr(), pos.data_ptr()
    a.qg_seq, a.qg_tok0, a.qg_ntok, a.o_part, a.ml_part = idx.data_ptr(), idx.data_ptr(), one.data_ptr(), op.data_ptr(), mp.data_ptr()
    a.gate_src, a.out, a.hq, a.hkv, a.max_blocks, a.nsplit = gg.data_ptr(), out.data_ptr(), H, hkv, nb, ns
    a.ld, a.num_qg, a.scale_log2e, a.num_blocks = ld, S, D ** -0.5 * math.log2(math.e), S * nb
    rows.append(_row(f"decode: attention over {ctx} keys, {G} heads per KV head (other model)", timed(lambda: F.attn_paged(a, D)),
                     flops=4 * S * H * ctx * D, nbytes=4 * S * ctx * hkv * D))
    return rows


def run(args) -> dict:
    from tileinfer_b200.models.kabadra import KABADRA_2K, KABADRA_4K
    hbm, tf, basis = peaks()
    res = {"metric": "kabadra_tok_s", "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "higher_is_better": True,
           "dtype": "bf16", "data": "synthetic: random tokens, random weights", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "basis": basis},
           "sizes": {}}
    for cfg, prompt, ctx in ((KABADRA_2K, 8192, 2048), (KABADRA_4K, 8192, 4096)):
        rows = kernels(cfg, prompt, ctx, 64)
        torch.cuda.empty_cache()
        ours = throughput(cfg, prompt, ctx, (1, 16, 64), args.steps, args.warmup)
        other = throughput(closest(cfg), prompt, ctx, (1, 16, 64), args.steps, args.warmup)
        res["sizes"][cfg.name] = {"layers": cfg.num_layers, "prompt": prompt, "context": ctx, "kabadra": ours, "attention_model": other, "kernels": rows}
        torch.cuda.empty_cache()
    res["value"] = res["sizes"]["kabadra-4k"]["kabadra"]["decode_64_tok_s"]
    res["config"] = {"model": "kabadra-4k", "global_batch": 64, "parallelism": "tp1", "cuda_graph": True,
                     "l2": "kernels: flushed between iterations; steps: more weights than L2"}
    return res


def table(res) -> str:
    lines = []
    for name, s in res["sizes"].items():
        lines.append(f"## {name}: {s['layers']} layers, prompt {s['prompt']}, decode context {s['context']}")
        keys = [k for k in s["kabadra"] if k.endswith("tok_s")]
        lines += [f"{k:20s} kabadra {s['kabadra'][k]:>12} other {s['attention_model'][k]:>12}" for k in keys]
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
