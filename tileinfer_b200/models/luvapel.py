"""Luvapel: configuration, checkpoint and random weights.

A decoder whose sublayers read the fp32 residual itself; what a sublayer gives is gated element by element (sigmoid of a
projection of its input), normed and added.  A layer's mixer is one of

  parallel       two mixers on the same input, each normed over the width, averaged: windowed attention (values are the key
                 projections, heads normed one by one, rotation of neighbouring dimensions, a temperature per head, a gate per
                 output dimension), and the gated delta rule (short convolutions, one decay and one step per head, gated head norm)
  general_delta  the generalized delta rule: a decay and a removal rate per key channel, gated head norm

and its feed-forward the square of a rectified product, or none.  A layer may run on the tensors of another one with a cache
and state of its own.

config.json:  architecture "Luvapel", vocab, width, norm.eps, embedding.scale, and `layers`, a list of
{type, mixer, mlp or null, weights_of?}:
  parallel:       {left: {heads, kv_heads, dim, vdim, rot: {base, dims}, scale, mask: {size}}, right: {heads, kv_heads, dim, vdim, conv}}
  general_delta:  {heads, dim}; the rank of the decay's product is the number of rows of mix.w1
  mlp:            {kind: "dense", ff}
Tensors:  embed, final.norm, head; per layer that owns tensors l<i>.{norm1, rg1, rg1.b} and with a feed-forward
l<i>.{norm2, rg2, rg2.b, mlp.up, mlp.down}; l<i>.mix.left.{q, k, q.norm, k.norm, temp, g, o, out} and
l<i>.mix.right.{q, k, v (each with .conv), b, a, A_log, dt_bias, g, norm, o, out}, or l<i>.mix.{r, k, v, g, a, a.b, w1, w2, w0, norm, o}.
Matrices are [out, in], convolutions [channels, taps].
"""
from __future__ import annotations

import math
import os
from dataclasses import dataclass, replace

from .checkpoint import make_source, stored_shapes

ARCHITECTURE = "Luvapel"
DECAY_SCALE = math.exp(-0.5)            # the general rule's log decay is this times minus a sigmoid
BRANCH_SCALE = 0.5                      # of the two halves of a parallel mixer


@dataclass(frozen=True)
class KeyValueAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int                           # equal to dim: the values are the key projections
    rot_base: float
    rot_dims: int
    scale: float
    window: int                         # positions seen, the token itself included


@dataclass(frozen=True)
class GatedDelta:
    heads: int
    kv_heads: int                       # heads of queries and keys
    dim: int
    vdim: int
    taps: int                           # of the convolutions over time


@dataclass(frozen=True)
class ParallelMixer:
    left: KeyValueAttention
    right: GatedDelta


@dataclass(frozen=True)
class GeneralDelta:
    heads: int
    dim: int
    decay_rank: int = 16                # inner size of the decay's two-matrix product


@dataclass(frozen=True)
class SquaredRelu:
    ff: int


@dataclass(frozen=True)
class LuvapelLayer:
    mixer: ParallelMixer | GeneralDelta
    mlp: SquaredRelu | None
    weights_of: int | None = None       # layer whose tensors this one uses; None: its own


@dataclass(frozen=True)
class LuvapelConfig:
    name: str
    vocab_size: int
    hidden_size: int
    layers: tuple
    rms_eps: float
    embedding_scale: float
    max_position_embeddings: int = 1 << 20     # no table of positions: a bound for buffers only
    eos_token_ids: tuple = ()

    family = "luvapel"
    recurrent = True                    # every layer has a recurrent state

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def num_attn_layers(self) -> int:
        return sum(isinstance(L.mixer, ParallelMixer) for L in self.layers)

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        j = self.layers[i].weights_of
        return i if j is None else j

    def validate(self) -> "LuvapelConfig":
        def need(ok, i, what):
            if not ok:
                raise ValueError(f"layer {i}: bad sizes ({what})")

        if min(self.vocab_size, self.hidden_size) < 1 or not self.layers:
            raise ValueError("vocabulary, width and layers must not be empty")
        for i, L in enumerate(self.layers):
            m, j = L.mixer, L.weights_of
            if j is not None:
                if not 0 <= j < len(self.layers) or self.layers[j].weights_of is not None:
                    raise ValueError(f"layer {i}: weights_of must name a layer with tensors of its own, got {j}")
                if replace(L, weights_of=None) != self.layers[j]:
                    raise ValueError(f"layer {i} uses the tensors of layer {j} but is not equal to it")
            if isinstance(m, ParallelMixer):
                a, r = m.left, m.right
                need(min(a.heads, a.kv_heads, a.dim, a.window) >= 1 and a.heads % a.kv_heads == 0, i, a)
                need(a.vdim == a.dim, i, f"values are keys: {a}")
                need(a.rot_dims % 2 == 0 and 0 <= a.rot_dims <= a.dim, i, a)
                need(min(r.heads, r.kv_heads, r.dim, r.vdim, r.taps) >= 1 and r.heads % r.kv_heads == 0, i, r)
            else:
                need(min(m.heads, m.dim, m.decay_rank) >= 1, i, m)
            need(L.mlp is None or L.mlp.ff >= 1, i, L.mlp)
        return self

    def validate_tp(self, tp: int) -> None:
        if tp > 1:
            raise ValueError("Luvapel runs on one GPU (tp_size = 1)")

    # ---- file format
    @classmethod
    def from_dict(cls, d: dict, name: str = ARCHITECTURE, decay_rank=None) -> "LuvapelConfig":
        """`decay_rank`: layer -> rank of its decay product (the tensors carry it, not the file)."""
        if d.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} config: architecture {d.get('architecture')!r}")
        layers = []
        for i, e in enumerate(d["layers"]):
            j = None if e.get("weights_of") is None else int(e["weights_of"])
            mixer = _mixer(i, e["type"], e["mixer"], (decay_rank or {}).get(i if j is None else j))
            layers.append(LuvapelLayer(mixer, _mlp(i, e.get("mlp")), j))
        return cls(name=name, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=tuple(layers),
                   rms_eps=float(d["norm"]["eps"]), embedding_scale=float(d["embedding"]["scale"])).validate()

    def to_dict(self) -> dict:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.rms_eps},
                "embedding": {"scale": self.embedding_scale}, "layers": [_layer_dict(L) for L in self.layers]}

    # ---- tensors
    def tensor_shapes(self) -> dict:
        W, V = self.hidden_size, self.vocab_size
        s = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
        for i, L in enumerate(self.layers):
            if L.weights_of is not None:
                continue
            m, p = L.mixer, f"l{i}."
            s[p + "norm1"], s[p + "rg1"], s[p + "rg1.b"] = (W,), (W, W), (W,)
            if L.mlp is not None:
                s[p + "norm2"], s[p + "rg2"], s[p + "rg2.b"] = (W,), (W, W), (W,)
                s[p + "mlp.up"], s[p + "mlp.down"] = (L.mlp.ff, W), (W, L.mlp.ff)
            p += "mix."
            if isinstance(m, GeneralDelta):
                n = m.heads * m.dim
                for t in ("r", "k", "v", "g", "a"):
                    s[p + t] = (n, W)
                s[p + "a.b"] = s[p + "w0"] = s[p + "norm"] = (n,)
                s[p + "w1"], s[p + "w2"], s[p + "o"] = (m.decay_rank, W), (n, m.decay_rank), (W, n)
                continue
            a, r, q = m.left, m.right, p + "left."
            s[q + "q"], s[q + "k"], s[q + "g"] = (a.heads * a.dim, W), (a.kv_heads * a.dim, W), (a.heads * a.vdim, W)
            s[q + "q.norm"] = s[q + "k.norm"] = (a.dim,)
            s[q + "temp"], s[q + "o"], s[q + "out"] = (a.heads,), (W, a.heads * a.vdim), (W,)
            q = p + "right."
            for t, rows in (("q", r.kv_heads * r.dim), ("k", r.kv_heads * r.dim), ("v", r.heads * r.vdim)):
                s[q + t], s[f"{q}{t}.conv"] = (rows, W), (rows, r.taps)
            s[q + "a"] = s[q + "b"] = (r.heads, W)
            s[q + "A_log"] = s[q + "dt_bias"] = (r.heads,)
            s[q + "g"], s[q + "norm"] = (r.heads * r.vdim, W), (r.vdim,)
            s[q + "o"], s[q + "out"] = (W, r.heads * r.vdim), (W,)
        return s


def _mixer(i: int, kind: str, m: dict, rank):
    if kind == "general_delta":
        g = GeneralDelta(heads=int(m["heads"]), dim=int(m["dim"]))
        return g if rank is None else replace(g, decay_rank=int(rank))
    if kind != "parallel":
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    a, r = m["left"], m["right"]
    return ParallelMixer(
        KeyValueAttention(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                          rot_base=float(a["rot"]["base"]), rot_dims=int(a["rot"]["dims"]), scale=float(a["scale"]), window=int(a["mask"]["size"])),
        GatedDelta(heads=int(r["heads"]), kv_heads=int(r["kv_heads"]), dim=int(r["dim"]), vdim=int(r["vdim"]), taps=int(r["conv"])))


def _mlp(i: int, f: dict | None):
    if f is None:
        return None
    if f["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
    return SquaredRelu(int(f["ff"]))


def _layer_dict(L: LuvapelLayer) -> dict:
    m = L.mixer
    if isinstance(m, GeneralDelta):
        e = {"type": "general_delta", "mixer": {"heads": m.heads, "dim": m.dim}}
    else:
        a, r = m.left, m.right
        e = {"type": "parallel", "mixer": {
            "left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "rot": {"base": a.rot_base, "dims": a.rot_dims},
                     "scale": a.scale, "mask": {"size": a.window}},
            "right": {"heads": r.heads, "kv_heads": r.kv_heads, "dim": r.dim, "vdim": r.vdim, "conv": r.taps}}}
    e["mlp"] = None if L.mlp is None else {"kind": "dense", "ff": L.mlp.ff}
    if L.weights_of is not None:
        e["weights_of"] = L.weights_of
    return e


# --------------------------------------------------------------------------- presets
def _parallel(heads, kv, dim, window, delta_heads, delta_kv, delta_dim, delta_vdim):
    left = KeyValueAttention(heads=heads, kv_heads=kv, dim=dim, vdim=dim, rot_base=5e5, rot_dims=dim, scale=dim ** -0.5, window=window)
    return ParallelMixer(left, GatedDelta(heads=delta_heads, kv_heads=delta_kv, dim=delta_dim, vdim=delta_vdim, taps=4))


def stack(mixers: tuple, mlp: SquaredRelu, repeats: int, shared: int = 0) -> tuple:
    """`repeats` times the mixers, each with tensors of its own, then `shared` more rounds on the tensors of the first."""
    own = tuple(LuvapelLayer(m, mlp) for m in mixers) * repeats
    return own + tuple(replace(L, weights_of=i) for _ in range(shared) for i, L in enumerate(own[:len(mixers)]))


TINY = LuvapelConfig(
    name="tiny-luvapel", vocab_size=1024, hidden_size=192, rms_eps=1e-6, embedding_scale=192 ** 0.5, max_position_embeddings=8192,
    layers=stack((_parallel(6, 2, 32, 70, 4, 2, 24, 48), GeneralDelta(3, 40, 12)), SquaredRelu(288), 1, shared=1)
    + (LuvapelLayer(GeneralDelta(2, 64, 8), None),), eos_token_ids=(1023,))

# Layers of the size of a few-billion and a ten-billion-parameter model; the benchmark takes as many as it needs.
LUVAPEL_2K = LuvapelConfig(
    name="luvapel-2k", vocab_size=65536, hidden_size=2048, rms_eps=1e-6, embedding_scale=2048 ** 0.5, max_position_embeddings=32768,
    layers=stack((_parallel(16, 4, 128, 1024, 16, 8, 128, 128), GeneralDelta(16, 128, 64), GeneralDelta(16, 128, 64)), SquaredRelu(6144), 2))
LUVAPEL_4K = LuvapelConfig(
    name="luvapel-4k", vocab_size=65536, hidden_size=4096, rms_eps=1e-6, embedding_scale=64.0, max_position_embeddings=32768,
    layers=stack((_parallel(32, 8, 128, 4096, 32, 16, 128, 128), GeneralDelta(32, 128, 64), GeneralDelta(32, 128, 64)), SquaredRelu(12288), 2))

PRESETS = {c.name: c for c in (TINY, LUVAPEL_2K, LUVAPEL_4K)}


def load_config(model_dir: str, d: dict) -> LuvapelConfig:
    rank = {int(n[1:n.index(".")]): s[0] for n, s in stored_shapes(model_dir).items() if n.startswith("l") and n.endswith(".mix.w1")}
    return LuvapelConfig.from_dict(d, name=os.path.basename(os.path.normpath(model_dir)) or ARCHITECTURE, decay_rank=rank)


def _random_scale(name: str, shape) -> float:
    """Matrices are scaled by their input size, convolutions by their taps, embeddings too (the configuration scales them up
    again); the vectors of the recurrences and the gates' biases are N(0, 1/4), temperatures and branch norms N(0, 1)."""
    if name.endswith((".dt_bias", ".A_log", ".w0", ".b")) and len(shape) == 1:
        return 0.5
    return 1.0 if len(shape) == 1 else shape[-1] ** -0.5


def make_weights(cfg: LuvapelConfig, spec: str, model_dir: str | None, device="cpu"):
    return make_source(cfg, spec, model_dir, device, _random_scale)
