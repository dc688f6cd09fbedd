"""Small Gerivik configurations for the tests: sizes that are no multiples of anything the kernels like, layers that differ
from each other, groups of one and of all experts, layers on another layer's tensors."""
import torch

import gerivik_oracle as oracle
from kabadra_cases import cut, engine, replay, rms_error, tokens  # noqa: F401  (engine and schedule helpers)



def moe(experts, top, ff, limit, identity=0, count=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": count, "keep": keep}}}


def attention(heads, kv, dim, vdim, rot, mlp=None, base=700.0, scale=None, softcap=6.0):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "softcap": softcap,
                                                       "rot": {"base": base, "dims": rot}, "scale": 2.0 * dim ** -0.5 if scale is None else scale}}


def gla(heads, dim, vdim, tau=5.0, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def again(layers, i):
    """The entry of a layer that runs on the tensors of layer i."""
    return dict(layers[i], weights_of=i)


def config(layers, width=136, vocab=331, eps=1e-5, scale=3.0):
    return {"architecture": "Gerivik", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}}


_A = [
    gla(3, 24, 40, 3.0, moe(6, 3, 40, 0.8, identity=2, count=4, keep=2)),
    attention(6, 2, 40, 24, 18),
    gla(1, 72, 136, 1.0, moe(5, 1, 72, 2.5)),
    attention(4, 4, 16, 72, 16, moe(3, 2, 24, 0.5, identity=6, count=3, keep=1), softcap=1.5),
]
MIXED = config(_A + [again(_A, 0), again(_A, 1), again(_A, 3)])
# more query heads per key head than a block takes (prime and not), heads padded to the widest tensor-core form
GROUPS = config([attention(34, 2, 20, 130, 6, moe(20, 5, 32, 1.0, identity=4, count=6, keep=5)), gla(2, 130, 64, 16.0, moe(70, 9, 16, 3.0, identity=10, count=8, keep=3)),
                 attention(40, 2, 130, 24, 130)], width=192, vocab=512, eps=1e-3, scale=11.0)
# heads wider than the tensor-core attention and the chunked recurrence take
WIDE_HEADS = config([attention(2, 1, 264, 300, 40, moe(2, 2, 16, 4.0)), gla(1, 300, 24, 2.0), gla(2, 200, 72, 30.0)], width=48, vocab=140)
ONE = config([gla(2, 32, 24, 7.0, moe(7, 2, 24, 1.5, identity=1, count=2, keep=1)), attention(4, 2, 32, 40, 8, moe(4, 2, 24, 1.5), base=2e5)],
             width=96, vocab=270)
# recurrence only: no pages are ever read
STATE_ONLY = config([gla(2, 48, 48, 0.3), gla(3, 64, 64, 16.0, moe(4, 2, 32, 1.0))], width=64, vocab=97)
CASES = {"mixed": MIXED, "groups": GROUPS, "wide_heads": WIDE_HEADS, "one": ONE, "state_only": STATE_ONLY}
RANKS = {"mixed": {0: 5, 2: 33}, "groups": {1: 16}, "wide_heads": {1: 1, 2: 40}}


def model(tmp_path, name, seed=3, decisive=False):
    """(folder, cfg, weights) of a case, written as a checkpoint.  `decisive`: corrections so far apart that every token
    chooses the same experts, whatever the precision of its scores."""
    cfg = CASES[name] if isinstance(name, str) else name
    rank = None
    if isinstance(name, str):
        rank = {i: RANKS.get(name, {}).get(i, 8) for i in range(len(cfg["layers"]))}
    w = oracle.random_weights(cfg, seed, rank)
    if decisive:
        g = torch.Generator().manual_seed(seed)
        for n in w:
            if n.endswith(".correction"):
                w[n] = (-0.75 * torch.randperm(len(w[n]), generator=g)).to(torch.bfloat16)
            elif n.endswith(".router"):
                w[n] = (w[n].float() * 0.2).to(torch.bfloat16)
    return oracle.write_model(str(tmp_path / "model"), cfg, w), cfg, w


def quantised(weights):
    """What the int8 mode computes with: symmetric int8 per output row, scale rounded to bf16, on projections and experts."""
    out = {}
    for n, w in weights.items():
        if n.endswith((".q", ".k", ".v", ".g", ".o", ".a1", ".gate", ".up", ".down")):
            w = w.float()
            s = (w.abs().amax(1).clamp_min(1e-8) / 127.0).to(torch.bfloat16).float()[:, None]
            w = (w / s).round().clamp(-128, 127) * s
        out[n] = w
    return out


def errors(got, want):
    """Error of every position: root mean square of the difference (mean over the vocabulary taken off) over that of the
    wanted logits."""
    d, w = got.float() - want.float(), want.float() - want.float().mean(-1, keepdim=True)
    return (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()


def assert_close(got, want, quant):
    """32-bit: every position to 1e-4.  16-bit: about a hundredth at most positions; where a head's output nearly cancels
    its norm scales the rounding up again, so single positions may be several times worse (a bf16 run of the same equations
    shows the same)."""
    e = errors(got, want)
    if quant == "fp32":
        assert e.max() < 1e-4, float(e.max())
    else:
        q = [float(e.quantile(x)) for x in (0.5, 0.9, 1.0)]
        assert q[0] < 0.02 and q[1] < 0.04 and q[2] < 0.15, q
