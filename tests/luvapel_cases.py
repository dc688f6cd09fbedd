"""Small Luvapel configurations for the tests: sizes that are no multiples of anything the kernels like, layers that differ from
each other, tensors shared between layers, windows of one token and of several tiles, convolutions of one to five taps, ranks of
the decay below and above a warp."""
import luvapel_oracle as oracle
from gerivik_cases import assert_close, errors  # noqa: F401  (comparison helpers)
from kabadra_cases import cut, engine, replay, rms_error, tokens  # noqa: F401  (engine and schedule helpers)


def attention(heads, kv, dim, rot, window, base=900.0, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "rot": {"base": base, "dims": rot},
            "scale": 1.2 * dim ** -0.5 if scale is None else scale, "mask": {"size": window}}


def gated(heads, kv, dim, vdim, taps):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": taps}


def parallel(left, right, ff=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def general(heads, dim, ff=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=136, vocab=331, eps=1e-5, scale=9.0, shared=()):
    """`shared`: layers after the given ones that run on the tensors of those listed."""
    layers = list(layers) + [dict(layers[j], weights_of=j) for j in shared]
    return {"architecture": "Luvapel", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}}


MIXED = config([
    parallel(attention(6, 2, 40, 18, 33), gated(6, 2, 24, 40, 4), ff=72),
    general(3, 24, ff=40),
    parallel(attention(3, 3, 24, 24, 1), gated(4, 4, 72, 20, 1)),
    general(1, 70),
    parallel(attention(4, 1, 72, 2, 100, base=2e4), gated(3, 1, 40, 136, 5), ff=200),
], width=152, shared=(1, 0))
# more query heads per key head than a block takes, windows over several tiles, the widest tensor-core forms
WIDE = config([
    parallel(attention(34, 2, 128, 64, 200), gated(10, 5, 130, 64, 3), ff=96),
    general(2, 130, ff=64),
    parallel(attention(2, 1, 200, 100, 129, scale=0.05), gated(2, 1, 64, 200, 2), ff=64),
    general(5, 64),
], width=192, vocab=512, eps=1e-3, scale=1.0)
# heads and states beyond what the tiled and the chunked kernels take
LARGE = config([
    parallel(attention(2, 1, 264, 100, 90), gated(2, 1, 300, 24, 7), ff=32),
    general(1, 260, ff=16),
], width=48, vocab=140)
ONE = config([
    parallel(attention(4, 2, 32, 8, 40, base=2e4), gated(4, 2, 32, 24, 4), ff=48),
    general(2, 40, ff=56),
], width=96, vocab=270, shared=(0,))
# no attention: a sequence is its states
RECURRENT = config([general(3, 32, ff=64), general(2, 24)], width=64, vocab=97, shared=(0, 0))
CASES = {"mixed": MIXED, "wide": WIDE, "large": LARGE, "one": ONE, "recurrent": RECURRENT}
RANKS = {"mixed": 5, "wide": 40, "large": 33, "one": 16, "recurrent": 1}


def model(tmp_path, name, seed=3, rank=16):
    """(folder, cfg, weights) of a case, written as a checkpoint."""
    cfg = CASES[name] if isinstance(name, str) else name
    w = oracle.random_weights(cfg, seed, RANKS.get(name, rank) if isinstance(name, str) else rank)
    return oracle.write_model(str(tmp_path / "model"), cfg, w), cfg, w


def quantised(weights):
    """What the int8 mode computes with: symmetric int8 per output row, scale rounded to bf16, on the projections."""
    out = {}
    for n, w in weights.items():
        if w.dim() == 2 and n.endswith((".q", ".k", ".v", ".g", ".o", ".r", ".a", ".b", ".w1", ".rg1", ".rg2", ".up", ".down")):
            w = w.float()
            s = (w.abs().amax(1).clamp_min(1e-8) / 127.0).bfloat16().float()[:, None]
            w = (w / s).round().clamp(-128, 127) * s
        out[n] = w
    return out
