"""Small Kabadra configurations for the tests: sizes that are no multiples of anything the kernels like, layers that differ
from each other, and helpers that run requests through the engine step by step."""
import torch

import kabadra_oracle as oracle


def layer(heads, dim, vdim, kv_rank, window, scale=None, kv_from=None, ff=None, limit=1.0):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
         "scale": dim ** -0.5 if scale is None else scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers, width=136, vocab=331, max_positions=700, eps=1e-5, logit_scale=0.7):
    return {"architecture": "Kabadra", "layers": layers, "width": width, "vocab": vocab, "max_positions": max_positions,
            "norm": {"eps": eps}, "logit_scale": logit_scale}


# layers of unequal head counts, sizes and windows; a layer without feed-forward; latents shared over several layers by
# readers whose windows are larger and smaller than the owner's
MIXED = config([
    layer(3, 24, 40, 56, 17, ff=100, limit=0.8),
    layer(5, 40, 24, 130, 64, ff=72, limit=2.5),
    layer(2, 72, 8, 56, 41, kv_from=0, scale=0.21),
    layer(4, 16, 96, 130, 5, kv_from=1, ff=136, limit=1.3),
    layer(1, 8, 16, 56, 1, kv_from=0, ff=40, limit=0.3),
])
# one head group more than a block takes, a latent wider than one tile, a window over several tiles of keys
WIDE = config([
    layer(18, 32, 32, 200, 300, ff=96, limit=3.0),
    layer(20, 48, 64, 200, 150, kv_from=0, ff=160, limit=1.1),
], width=192, vocab=512, logit_scale=1.3, eps=1e-3)
ONE = config([layer(2, 32, 24, 40, 23, scale=0.4, ff=64, limit=1.5)], width=96, vocab=270, logit_scale=1.0)
# latents of the sizes that the widest kernels serve
DEEP_RANK = config([layer(4, 64, 64, 512, 130, ff=128, limit=2.0), layer(33, 16, 16, 512, 70, kv_from=0),
                    layer(2, 64, 128, 640, 90, ff=64, limit=1.0)], width=256, vocab=300)
# heads wider than the tiled prefill kernel takes: every token goes through the split attention
WIDE_HEADS = config([layer(2, 264, 280, 24, 40, ff=32), layer(1, 16, 300, 24, 90, kv_from=0)], width=48, vocab=140)
CASES = {"wide_heads": WIDE_HEADS, "mixed": MIXED, "wide": WIDE, "one": ONE, "deep_rank": DEEP_RANK}


def tokens(cfg, n, seed=0):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def quantised(weights):
    """What the int8 mode computes with: symmetric int8 per output row, scale rounded to bf16, on the projections."""
    out = {}
    for n, w in weights.items():
        if n.endswith((".q", ".dkv", ".g", ".o", ".gate", ".up", ".down")):
            w = w.float()
            s = (w.abs().amax(1).clamp_min(1e-8) / 127.0).to(torch.bfloat16).float()[:, None]
            w = (w / s).round().clamp(-128, 127) * s
        out[n] = w
    return out


def rms_error(got, want):
    """Root mean square of the difference (mean over the vocabulary taken off) over that of the wanted logits."""
    d = got.float() - want.float()
    d = d - d.mean(-1, keepdim=True)
    w = want.float() - want.float().mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()).max().item()


def engine(folder, quant, device, blocks=64, seqs=4, **kw):
    from tileinfer_b200.engine.llm_engine import LLMEngine
    kw.setdefault("enable_prefix_caching", False)
    return LLMEngine(str(folder), quantization=quant, device=device, num_kvcache_blocks=blocks, max_num_seqs=seqs, **kw)


def replay(eng, schedule, prompts):
    """Runs [[(request, tokens), ...], ...] and returns request -> logits of every position it ran; a request ends with its
    last token."""
    from tileinfer_b200.engine.replay import ReplaySession
    s, at, out = ReplaySession(eng), {}, {}
    for step in schedule:
        entries, ended = [], []
        for rid, n in step:
            lo = at.get(rid, 0)
            entries.append({"id": rid, "tokens": prompts[rid][lo:lo + n], "want": list(range(n))})
            at[rid] = lo + n
            if at[rid] == len(prompts[rid]):
                ended.append(rid)
        logits, row = s.step(entries, ended), 0
        for rid, n in step:
            out.setdefault(rid, []).append(logits[row:row + n].clone())
            row += n
    assert not s.live
    return {rid: torch.cat(v) for rid, v in out.items()}


def cut(rid, total, sizes):
    """A schedule of one request: portions of the given sizes in turn until all its tokens have run."""
    steps, done, k = [], 0, 0
    while done < total:
        n = min(sizes[k % len(sizes)], total - done)
        steps.append([(rid, n)])
        done, k = done + n, k + 1
    return steps


def model(tmp_path, name, seed=3, gain=1.0):
    """(folder, cfg, weights) of a case, written as a checkpoint."""
    cfg = CASES[name] if isinstance(name, str) else name
    w = oracle.random_weights(cfg, seed, gain)
    return oracle.write_model(str(tmp_path / "model"), cfg, w), cfg, w
