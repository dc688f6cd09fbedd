"""Small Nogidra configurations for the tests: sizes that are no multiples of anything the kernels like, layers that differ
from each other, group norms that cut heads in two, windows of one token and of several tiles, convolutions of one to five
taps."""
import nogidra_oracle as oracle
from gerivik_cases import assert_close, errors  # noqa: F401  (comparison helpers)
from kabadra_cases import cut, engine, replay, rms_error, tokens  # noqa: F401  (engine and schedule helpers)


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def attention(heads, kv, dim, vdim, taps, window, coef=0.4, every=7, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": taps, "q_temp": {"coef": coef, "every": every},
        "scale": 1.5 * dim ** -0.5 if scale is None else scale, "mask": {"size": window}}}


def latent(heads, dim, rot, vdim, rank, window, base=700.0, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": {"base": base, "dims": rot},
        "scale": 1.5 * (dim + rot) ** -0.5 if scale is None else scale, "mask": {"size": window}}}


def normed(heads, kv, dim, vdim, rot, window, base=900.0, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
            "scale": 1.2 * dim ** -0.5 if scale is None else scale, "mask": {"size": window}}


def ssm(heads, vdim, state, groups, taps, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": taps, "norm_groups": norm_groups}


def parallel(left, right, left_scale=0.6, right_scale=1.3, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left, "left_scale": left_scale, "right": right, "right_scale": right_scale}}


def config(layers, width=136, vocab=331, eps=1e-5, cap=9.0):
    return {"architecture": "Nogidra", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": cap}


MIXED = config([
    parallel(normed(6, 2, 40, 24, 18, 33), ssm(6, 20, 24, 3, 4, 4), mlp=moe(6, 3, 40)),
    attention(4, 4, 24, 40, 5, 17),
    latent(3, 24, 10, 40, 56, 21, mlp=dense(72)),
    attention(6, 2, 20, 8, 1, 64, coef=-0.1, every=1, mlp=moe(3, 3, 24)),
    parallel(normed(3, 1, 16, 72, 16, 100), ssm(4, 12, 70, 1, 2, 1), -0.7, 0.4, mlp=dense(40)),
    latent(5, 40, 24, 8, 130, 1, mlp=moe(20, 1, 16)),
    attention(2, 1, 72, 24, 3, 5, every=50, mlp=dense(136)),
], width=152)
# more query heads per key head than a block takes, windows over several tiles, the widest tensor-core forms
WIDE = config([
    latent(18, 48, 64, 64, 512, 150, mlp=dense(96)),
    parallel(normed(34, 2, 128, 24, 40, 200), ssm(10, 130, 130, 5, 3, 13), mlp=moe(70, 9, 16)),
    attention(40, 2, 24, 130, 4, 129, mlp=dense(160)),
    latent(33, 130, 62, 20, 194, 300),
], width=192, vocab=512, eps=1e-3, cap=30.0)
# heads, latents and states beyond what the tiled and the chunked kernels take
LARGE = config([
    latent(2, 260, 20, 300, 600, 40, mlp=dense(32)),
    parallel(normed(2, 1, 264, 24, 100, 90), ssm(2, 24, 300, 2, 4, 2), mlp=moe(2, 2, 16)),
    attention(1, 1, 24, 270, 7, 50),
], width=48, vocab=140)
ONE = config([
    parallel(normed(4, 2, 32, 40, 8, 40, base=2e4), ssm(2, 24, 32, 2, 4, 1), mlp=moe(7, 2, 24)),
    attention(4, 2, 32, 40, 3, 23, mlp=dense(48)),
    latent(2, 32, 16, 24, 40, 37, mlp=moe(4, 2, 24)),
], width=96, vocab=270)
# no recurrent layer: a sequence is its cache pages
LATENT_ONLY = config([latent(3, 32, 32, 16, 64, 50, mlp=dense(64)), latent(1, 16, 2, 24, 30, 70, mlp=moe(4, 1, 24))], width=64, vocab=97)
CASES = {"mixed": MIXED, "wide": WIDE, "large": LARGE, "one": ONE, "latent_only": LATENT_ONLY}


def model(tmp_path, name, seed=3, decisive=False):
    """(folder, cfg, weights) of a case, written as a checkpoint."""
    cfg = CASES[name] if isinstance(name, str) else name
    w = oracle.random_weights(cfg, seed, decisive)
    return oracle.write_model(str(tmp_path / "model"), cfg, w), cfg, w


def quantised(weights):
    """What the int8 mode computes with: symmetric int8 per output row, scale rounded to bf16, on projections and experts."""
    out = {}
    for n, w in weights.items():
        if n.endswith((".q", ".k", ".v", ".g", ".o", ".dkv", ".in", ".gate", ".up", ".down")):
            w = w.float()
            s = (w.abs().amax(1).clamp_min(1e-8) / 127.0).to(w.dtype).bfloat16().float()[:, None]
            w = (w / s).round().clamp(-128, 127) * s
        out[n] = w
    return out
