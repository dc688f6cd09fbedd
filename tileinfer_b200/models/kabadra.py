"""Kabadra: configuration, checkpoint reader and random weights.

A decoder whose layers are parallel (one norm, the mixer and the feed-forward both read it, both add to the fp32
residual).  The mixer is latent attention without positions: keys and values are linear maps of one cached latent per
token, inside a sliding window, with a sink per head in the softmax and a sigmoid gate per head on the output.  A layer
may reuse the latents another layer has cached.  Positions enter as learned vectors added to the token embedding.

config.json:  architecture "Kabadra", vocab, width, max_positions, norm.eps, logit_scale, and `layers`, a list of
{type, mixer: {heads, dim, vdim, kv_rank, scale, mask: {size}, kv_from?}, mlp: {kind, ff, limit} or null}.
Tensors:  embed, pos, embed.norm, final.norm, head; per layer l<i>.norm1, l<i>.mix.{q, dkv, dkv.norm, uk, uv, sink, g, o},
l<i>.mlp.{gate, up, down}; matrices are [out, in].
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass

from .checkpoint import CheckpointWeights, make_source

ARCHITECTURE = "Kabadra"
MIXERS = ("latent_attention",)
GLU_ALPHA, GLU_BIAS = 1.702, 1.0        # g sigmoid(alpha g) (u + bias): constants of the design's feed-forward


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int                         # positions seen, the token itself included
    kv_from: int | None = None          # layer whose cached latents this layer reads; None: its own


@dataclass(frozen=True)
class ClampedGlu:
    ff: int
    limit: float


@dataclass(frozen=True)
class KabadraLayer:
    mixer: LatentMixer
    mlp: ClampedGlu | None


@dataclass(frozen=True)
class KabadraConfig:
    name: str
    vocab_size: int
    hidden_size: int
    layers: tuple
    rms_eps: float
    logit_scale: float
    max_position_embeddings: int
    eos_token_ids: tuple = ()

    family = "kabadra"
    num_gdn_layers = 0                  # no recurrent state
    recurrent = False

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def num_attn_layers(self) -> int:
        return len(self.layers)

    def latent_layer(self, i: int) -> int:
        """The layer whose cache layer i attends to."""
        src = self.layers[i].mixer.kv_from
        return i if src is None else src

    @property
    def latent_owners(self) -> tuple:
        return tuple(i for i, L in enumerate(self.layers) if L.mixer.kv_from is None)

    def validate(self) -> "KabadraConfig":
        for i, L in enumerate(self.layers):
            m = L.mixer
            if min(m.heads, m.dim, m.vdim, m.kv_rank, m.window) < 1:
                raise ValueError(f"layer {i}: sizes must be positive ({m})")
            if m.kv_from is not None:
                if not 0 <= m.kv_from < i:
                    raise ValueError(f"layer {i}: kv_from must name an earlier layer, got {m.kv_from}")
                src = self.layers[m.kv_from].mixer
                if src.kv_from is not None or src.kv_rank != m.kv_rank:
                    raise ValueError(f"layer {i}: layer {m.kv_from} has no latents of rank {m.kv_rank} of its own")
        return self

    def validate_tp(self, tp: int) -> None:
        if tp > 1:
            raise ValueError("Kabadra runs on one GPU (tp_size = 1)")

    # ---- file format
    @classmethod
    def from_dict(cls, d: dict, name: str = ARCHITECTURE) -> "KabadraConfig":
        if d.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} config: architecture {d.get('architecture')!r}")
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            m, f = e["mixer"], e.get("mlp")
            if f is not None and f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
            layers.append(KabadraLayer(
                LatentMixer(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                            scale=float(m["scale"]), window=int(m["mask"]["size"]),
                            kv_from=None if m.get("kv_from") is None else int(m["kv_from"])),
                None if f is None else ClampedGlu(ff=int(f["ff"]), limit=float(f["limit"]))))
        return cls(name=name, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=tuple(layers),
                   rms_eps=float(d["norm"]["eps"]), logit_scale=float(d["logit_scale"]),
                   max_position_embeddings=int(d["max_positions"])).validate()

    def to_dict(self) -> dict:
        layers = []
        for L in self.layers:
            m = {"heads": L.mixer.heads, "dim": L.mixer.dim, "vdim": L.mixer.vdim, "kv_rank": L.mixer.kv_rank,
                 "scale": L.mixer.scale, "mask": {"size": L.mixer.window}}
            if L.mixer.kv_from is not None:
                m["kv_from"] = L.mixer.kv_from
            mlp = None if L.mlp is None else {"kind": "dense", "ff": L.mlp.ff, "limit": L.mlp.limit}
            layers.append({"type": MIXERS[0], "mixer": m, "mlp": mlp})
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "layers": layers,
                "norm": {"eps": self.rms_eps}, "logit_scale": self.logit_scale, "max_positions": self.max_position_embeddings}

    # ---- tensors
    def tensor_shapes(self) -> dict:
        W, V = self.hidden_size, self.vocab_size
        s = {"embed": (V, W), "pos": (self.max_position_embeddings, W), "embed.norm": (W,), "final.norm": (W,), "head": (V, W)}
        for i, L in enumerate(self.layers):
            m, p = L.mixer, f"l{i}."
            s[p + "norm1"] = (W,)
            s[p + "mix.q"] = (m.heads * m.dim, W)
            if m.kv_from is None:
                s[p + "mix.dkv"], s[p + "mix.dkv.norm"] = (m.kv_rank, W), (m.kv_rank,)
            s[p + "mix.uk"], s[p + "mix.uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
            s[p + "mix.sink"], s[p + "mix.g"] = (m.heads,), (m.heads, W)
            s[p + "mix.o"] = (W, m.heads * m.vdim)
            if L.mlp is not None:
                s[p + "mlp.gate"] = s[p + "mlp.up"] = (L.mlp.ff, W)
                s[p + "mlp.down"] = (W, L.mlp.ff)
        return s


def stack(num_layers: int, mixer: LatentMixer, mlp: ClampedGlu, share: int = 1) -> tuple:
    """Equal layers in groups of `share` that use the latents of the group's first layer."""
    from dataclasses import replace
    return tuple(KabadraLayer(replace(mixer, kv_from=None if i % share == 0 else i - i % share), mlp) for i in range(num_layers))


TINY = KabadraConfig(
    name="tiny-kabadra", vocab_size=1024, hidden_size=256, rms_eps=1e-6, logit_scale=0.75, max_position_embeddings=4096,
    layers=stack(4, LatentMixer(heads=6, dim=32, vdim=48, kv_rank=64, scale=32 ** -0.5, window=100), ClampedGlu(512, 4.0), share=2),
    eos_token_ids=(1023,))

# Layers of the size of a few-billion and a ten-billion-parameter model; the benchmark takes as many as it needs.
KABADRA_2K = KabadraConfig(
    name="kabadra-2k", vocab_size=65536, hidden_size=2048, rms_eps=1e-6, logit_scale=1.0, max_position_embeddings=32768,
    layers=stack(8, LatentMixer(heads=16, dim=128, vdim=128, kv_rank=512, scale=128 ** -0.5, window=1024), ClampedGlu(8192, 7.0), share=2))
KABADRA_4K = KabadraConfig(
    name="kabadra-4k", vocab_size=65536, hidden_size=4096, rms_eps=1e-6, logit_scale=1.0, max_position_embeddings=32768,
    layers=stack(8, LatentMixer(heads=32, dim=128, vdim=128, kv_rank=512, scale=128 ** -0.5, window=4096), ClampedGlu(14336, 7.0), share=2))

PRESETS = {c.name: c for c in (TINY, KABADRA_2K, KABADRA_4K)}


def load_config(model_dir: str, d: dict) -> KabadraConfig:
    return KabadraConfig.from_dict(d, name=os.path.basename(os.path.normpath(model_dir)) or ARCHITECTURE)


# --------------------------------------------------------------------------- weight sources
KabadraWeights = CheckpointWeights


def _random_scale(name: str, shape) -> float:
    """Matrices are scaled by their input size; sinks and embeddings are N(0, 1)."""
    return 1.0 if name.endswith((".sink", "embed", "pos")) else shape[-1] ** -0.5


def make_weights(cfg: KabadraConfig, spec: str, model_dir: str | None, device="cpu"):
    return make_source(cfg, spec, model_dir, device, _random_scale)


def read_config_json(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)
