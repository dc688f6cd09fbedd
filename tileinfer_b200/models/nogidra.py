"""Nogidra: configuration, checkpoint and random weights.

A pre-norm decoder on an fp32 residual with capped logits.  A layer's mixer is one of

  attention         windowed attention over queries, keys and values that went through a short causal convolution; queries
                    grow with the logarithm of their position, a key costs a slope per head times its distance, and a gate
                    per head scales the output
  latent_attention  windowed attention whose keys and values are linear maps of one cached latent per token, beside a
                    rotated key part that all heads share
  parallel          two mixers on the same input, added with a scale each: windowed attention (biases, one norm over all
                    query heads and one over all key heads, rotation of neighbouring dimensions) and a state-space mixer
                    (short convolution, a decaying state per head, gated group norm)

and its feed-forward a gated unit with biases, a mixture of such units, or none.

config.json:  architecture "Nogidra", vocab, width, norm.eps, logit_softcap, and `layers`, a list of {type, mixer, mlp or null}:
  attention:         {heads, kv_heads, dim, vdim, conv, q_temp: {coef, every}, scale, mask: {size}}
  latent_attention:  {heads, dim, rot_dim, vdim, kv_rank, rot: {base, dims}, scale, mask: {size}}
  parallel:          {left: {heads, kv_heads, dim, vdim, rot: {base, dims}, scale, mask: {size}}, left_scale,
                      right: {heads, vdim, state, groups, conv, norm_groups}, right_scale}
  mlp:               {kind: "dense", ff} or {kind: "moe", expert: {ff}, router: {experts, top}}
Tensors:  embed, final.norm, head; per layer l<i>.{norm1, norm2}; l<i>.mix.{q, k, v} with .conv each, {g, o};
l<i>.mix.{q, dkv, dkv.norm, uk, uv, o}; l<i>.mix.left.{q, k, v} with .b each, {q.norm, k.norm, o} and
l<i>.mix.right.{in, conv, conv.b, dt_bias, A_log, D, norm, o}; l<i>.mlp.{gate, up, down} with .b each, or
l<i>.mlp.router and l<i>.mlp.e<n>.{gate, up, down}.  Matrices are [out, in], convolutions [channels, taps].
"""
from __future__ import annotations

import os
from dataclasses import dataclass

from .checkpoint import make_source

ARCHITECTURE = "Nogidra"


@dataclass(frozen=True)
class ConvAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int                           # of the convolutions over time
    temp_coef: float                    # q *= 1 + coef ln(floor((p + 1) / every) + 1)
    temp_every: int
    scale: float
    window: int                         # positions seen, the token itself included

    def slopes(self) -> list:
        """What a step of distance costs, per head."""
        return [2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads)]


@dataclass(frozen=True)
class RotaryLatent:
    heads: int
    dim: int                            # unrotated query / key dimensions of a head; rot_dim rotated ones follow
    rot_dim: int
    vdim: int
    kv_rank: int
    rot_base: float
    scale: float
    window: int


@dataclass(frozen=True)
class NormedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_base: float
    rot_dims: int
    scale: float
    window: int


@dataclass(frozen=True)
class StateSpace:
    heads: int
    vdim: int
    state: int
    groups: int                         # of heads that share B and C
    taps: int
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_channels(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class ParallelMixer:
    left: NormedAttention
    right: StateSpace
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DenseGlu:
    ff: int


@dataclass(frozen=True)
class SoftmaxExperts:
    experts: int
    top: int
    ff: int

    identity = 0                        # no experts that return their input, no groups, no corrected choice
    groups = keep = 1

    @property
    def choices(self) -> int:
        return self.experts


@dataclass(frozen=True)
class NogidraLayer:
    mixer: ConvAttention | RotaryLatent | ParallelMixer
    mlp: DenseGlu | SoftmaxExperts | None


@dataclass(frozen=True)
class NogidraConfig:
    name: str
    vocab_size: int
    hidden_size: int
    layers: tuple
    rms_eps: float
    logit_softcap: float
    max_position_embeddings: int = 1 << 20     # no table of positions: a bound for buffers only
    eos_token_ids: tuple = ()

    family = "nogidra"

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def num_attn_layers(self) -> int:
        return len(self.layers)         # every layer has a paged cache

    @property
    def recurrent(self) -> bool:
        """Whether a sequence has more than cache pages: recurrent states, or the last inputs of a convolution."""
        return any(not isinstance(L.mixer, RotaryLatent) for L in self.layers)

    def validate(self) -> "NogidraConfig":
        def need(ok, i, what):
            if not ok:
                raise ValueError(f"layer {i}: bad sizes ({what})")

        if min(self.vocab_size, self.hidden_size) < 1 or not self.layers:
            raise ValueError("vocabulary, width and layers must not be empty")
        for i, L in enumerate(self.layers):
            m, f = L.mixer, L.mlp
            for a in ((m.left,) if isinstance(m, ParallelMixer) else (m,)):
                need(min(a.heads, a.dim, a.vdim, a.window) >= 1, i, a)
                if isinstance(a, RotaryLatent):
                    need(a.kv_rank >= 1 and a.rot_dim >= 0 and a.rot_dim % 2 == 0, i, a)
                else:
                    need(a.kv_heads >= 1 and a.heads % a.kv_heads == 0, i, a)
                if isinstance(a, NormedAttention):
                    need(a.rot_dims % 2 == 0 and 0 <= a.rot_dims <= a.dim, i, a)
                if isinstance(a, ConvAttention):
                    need(a.taps >= 1 and a.temp_every >= 1, i, a)
            if isinstance(m, ParallelMixer):
                r = m.right
                need(min(r.heads, r.vdim, r.state, r.groups, r.taps, r.norm_groups) >= 1 and r.heads % r.groups == 0
                     and r.inner % r.norm_groups == 0, i, r)
            if isinstance(f, DenseGlu):
                need(f.ff >= 1, i, f)
            elif f is not None:
                need(min(f.experts, f.ff, f.top) >= 1 and f.top <= f.experts, i, f)
        return self

    def validate_tp(self, tp: int) -> None:
        if tp > 1:
            raise ValueError("Nogidra runs on one GPU (tp_size = 1)")

    # ---- file format
    @classmethod
    def from_dict(cls, d: dict, name: str = ARCHITECTURE) -> "NogidraConfig":
        if d.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} config: architecture {d.get('architecture')!r}")
        layers = tuple(NogidraLayer(_mixer(i, e["type"], e["mixer"]), _mlp(i, e.get("mlp"))) for i, e in enumerate(d["layers"]))
        return cls(name=name, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers,
                   rms_eps=float(d["norm"]["eps"]), logit_softcap=float(d["logit_softcap"])).validate()

    def to_dict(self) -> dict:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.rms_eps},
                "logit_softcap": self.logit_softcap, "layers": [_layer_dict(L) for L in self.layers]}

    # ---- tensors
    def tensor_shapes(self) -> dict:
        W, V = self.hidden_size, self.vocab_size
        s = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
        for i, L in enumerate(self.layers):
            m, f, p = L.mixer, L.mlp, f"l{i}."
            s[p + "norm1"] = (W,)
            q = p + "mix."
            if isinstance(m, ConvAttention):
                for n, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                    s[q + n], s[q + n + ".conv"] = (rows, W), (rows, m.taps)
                s[q + "g"], s[q + "o"] = (m.heads, W), (W, m.heads * m.vdim)
            elif isinstance(m, RotaryLatent):
                s[q + "q"] = (m.heads * (m.dim + m.rot_dim), W)
                s[q + "dkv"], s[q + "dkv.norm"] = (m.kv_rank + m.rot_dim, W), (m.kv_rank,)
                s[q + "uk"], s[q + "uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
                s[q + "o"] = (W, m.heads * m.vdim)
            else:
                a, r = m.left, m.right
                for n, rows in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                    s[f"{q}left.{n}"], s[f"{q}left.{n}.b"] = (rows, W), (rows,)
                s[q + "left.q.norm"], s[q + "left.k.norm"] = (a.heads * a.dim,), (a.kv_heads * a.dim,)
                s[q + "left.o"] = (W, a.heads * a.vdim)
                s[q + "right.in"] = (r.inner + r.conv_channels + r.heads, W)
                s[q + "right.conv"], s[q + "right.conv.b"] = (r.conv_channels, r.taps), (r.conv_channels,)
                s[q + "right.dt_bias"] = s[q + "right.A_log"] = s[q + "right.D"] = (r.heads,)
                s[q + "right.norm"], s[q + "right.o"] = (r.inner,), (W, r.inner)
            if f is None:
                continue
            s[p + "norm2"], q = (W,), p + "mlp."
            if isinstance(f, DenseGlu):
                s[q + "gate"] = s[q + "up"] = (f.ff, W)
                s[q + "gate.b"] = s[q + "up.b"] = (f.ff,)
                s[q + "down"], s[q + "down.b"] = (W, f.ff), (W,)
            else:
                s[q + "router"] = (f.experts, W)
                for e in range(f.experts):
                    s[f"{q}e{e}.gate"] = s[f"{q}e{e}.up"] = (f.ff, W)
                    s[f"{q}e{e}.down"] = (W, f.ff)
        return s


def _normed(a: dict) -> NormedAttention:
    return NormedAttention(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                           rot_base=float(a["rot"]["base"]), rot_dims=int(a["rot"]["dims"]), scale=float(a["scale"]),
                           window=int(a["mask"]["size"]))


def _mixer(i: int, kind: str, m: dict):
    if kind == "attention":
        return ConvAttention(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                             taps=int(m["conv"]), temp_coef=float(m["q_temp"]["coef"]), temp_every=int(m["q_temp"]["every"]),
                             scale=float(m["scale"]), window=int(m["mask"]["size"]))
    if kind == "latent_attention":
        if int(m["rot"]["dims"]) != int(m["rot_dim"]):
            raise ValueError(f"layer {i}: the rotated part of a head turns as a whole, got {m['rot']['dims']} of {m['rot_dim']} dimensions")
        return RotaryLatent(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                            kv_rank=int(m["kv_rank"]), rot_base=float(m["rot"]["base"]), scale=float(m["scale"]),
                            window=int(m["mask"]["size"]))
    if kind == "parallel":
        r = m["right"]
        right = StateSpace(heads=int(r["heads"]), vdim=int(r["vdim"]), state=int(r["state"]), groups=int(r["groups"]),
                           taps=int(r["conv"]), norm_groups=int(r["norm_groups"]))
        return ParallelMixer(_normed(m["left"]), right, float(m["left_scale"]), float(m["right_scale"]))
    raise ValueError(f"layer {i}: unknown mixer {kind!r}")


def _mlp(i: int, f: dict | None):
    if f is None:
        return None
    if f["kind"] == "dense":
        return DenseGlu(int(f["ff"]))
    if f["kind"] == "moe":
        return SoftmaxExperts(experts=int(f["router"]["experts"]), top=int(f["router"]["top"]), ff=int(f["expert"]["ff"]))
    raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")


def _layer_dict(L: NogidraLayer) -> dict:
    m, f = L.mixer, L.mlp
    if isinstance(m, ConvAttention):
        kind = "attention"
        mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "conv": m.taps,
                 "q_temp": {"coef": m.temp_coef, "every": m.temp_every}, "scale": m.scale, "mask": {"size": m.window}}
    elif isinstance(m, RotaryLatent):
        kind = "latent_attention"
        mixer = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank,
                 "rot": {"base": m.rot_base, "dims": m.rot_dim}, "scale": m.scale, "mask": {"size": m.window}}
    else:
        kind, a, r = "parallel", m.left, m.right
        mixer = {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim,
                          "rot": {"base": a.rot_base, "dims": a.rot_dims}, "scale": a.scale, "mask": {"size": a.window}},
                 "left_scale": m.left_scale,
                 "right": {"heads": r.heads, "vdim": r.vdim, "state": r.state, "groups": r.groups, "conv": r.taps,
                           "norm_groups": r.norm_groups},
                 "right_scale": m.right_scale}
    if f is None:
        mlp = None
    elif isinstance(f, DenseGlu):
        mlp = {"kind": "dense", "ff": f.ff}
    else:
        mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# --------------------------------------------------------------------------- presets
def _conv(heads, kv, dim, window):
    return ConvAttention(heads=heads, kv_heads=kv, dim=dim, vdim=dim, taps=4, temp_coef=0.25, temp_every=512, scale=dim ** -0.5, window=window)


def _latent(heads, dim, rot, rank, window):
    return RotaryLatent(heads=heads, dim=dim, rot_dim=rot, vdim=dim, kv_rank=rank, rot_base=1e5, scale=(dim + rot) ** -0.5, window=window)


def _parallel(heads, kv, dim, window, ssm_heads, ssm_vdim, state):
    left = NormedAttention(heads=heads, kv_heads=kv, dim=dim, vdim=dim, rot_base=1e5, rot_dims=dim, scale=dim ** -0.5, window=window)
    right = StateSpace(heads=ssm_heads, vdim=ssm_vdim, state=state, groups=2, taps=4, norm_groups=4)
    return ParallelMixer(left, right, 0.75, 0.9)


def _stack(mixers: tuple, dense: DenseGlu, moe: SoftmaxExperts, repeats: int) -> tuple:
    """Mixers in turn; every other layer has experts."""
    return tuple(NogidraLayer(m, moe if (r * len(mixers) + i) % 2 else dense) for r in range(repeats) for i, m in enumerate(mixers))


TINY = NogidraConfig(
    name="tiny-nogidra", vocab_size=1024, hidden_size=192, rms_eps=1e-6, logit_softcap=25.0, max_position_embeddings=8192,
    layers=_stack((_parallel(6, 2, 32, 70, 4, 48, 24), _conv(6, 3, 48, 50), _latent(3, 48, 16, 80, 90)), DenseGlu(288),
                  SoftmaxExperts(experts=12, top=3, ff=72), 1) + (NogidraLayer(_conv(3, 1, 64, 33), None),),
    eos_token_ids=(1023,))

# Layers of the size of a few-billion and a ten-billion-parameter model; the benchmark takes as many as it needs.
NOGIDRA_2K = NogidraConfig(
    name="nogidra-2k", vocab_size=65536, hidden_size=2048, rms_eps=1e-6, logit_softcap=30.0, max_position_embeddings=32768,
    layers=_stack((_latent(16, 128, 64, 512, 1024), _parallel(16, 4, 128, 1024, 32, 64, 128), _conv(16, 4, 128, 1024)), DenseGlu(6144),
                  SoftmaxExperts(experts=64, top=8, ff=768), 2))
NOGIDRA_4K = NogidraConfig(
    name="nogidra-4k", vocab_size=65536, hidden_size=4096, rms_eps=1e-6, logit_softcap=30.0, max_position_embeddings=32768,
    layers=_stack((_latent(32, 128, 64, 512, 4096), _parallel(32, 8, 128, 4096, 64, 64, 128), _conv(32, 8, 128, 4096)), DenseGlu(12288),
                  SoftmaxExperts(experts=64, top=8, ff=1536), 2))

PRESETS = {c.name: c for c in (TINY, NOGIDRA_2K, NOGIDRA_4K)}


def load_config(model_dir: str, d: dict) -> NogidraConfig:
    return NogidraConfig.from_dict(d, name=os.path.basename(os.path.normpath(model_dir)) or ARCHITECTURE)


def _random_scale(name: str, shape) -> float:
    """Matrices are scaled by their input size, convolutions by their taps; embeddings and the state-space vectors are
    N(0, 1)."""
    if name == "embed" or name.endswith((".dt_bias", ".A_log", ".D")):
        return 1.0
    return 0.1 if name.endswith(".b") else shape[-1] ** -0.5


def make_weights(cfg: NogidraConfig, spec: str, model_dir: str | None, device="cpu"):
    # the layers' norms are stored around zero, those inside mixers are plain factors
    return make_source(cfg, spec, model_dir, device, _random_scale, zero_norm=lambda name: ".mix." not in name)
