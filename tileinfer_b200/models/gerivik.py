"""Gerivik: configuration, checkpoint and random weights.

A decoder with a norm before and after every sublayer on an fp32 residual.  A layer's mixer is either causal softmax
attention (rotary positions on part of a head, then queries and keys divided by their own root mean square, scores capped
by a scaled tanh) or gated linear attention (a decaying state per head, one decay per key channel and token).  The
feed-forward is a mixture of experts: a softmax router over experts and identity experts, chosen inside the best groups
by corrected scores, weighted by the scores themselves.  A layer may run on the tensors of an earlier one with a cache or
state of its own.

config.json:  architecture "Gerivik", vocab, width, norm.eps, embedding.scale, and `layers`, a list of
{type: "attention" | "gla", mixer, mlp or null, weights_of?}:
  attention: {heads, kv_heads, dim, vdim, rot: {base, dims}, scale, softcap}
  gla:       {heads, dim, vdim, tau}; the rank of the decay's product is the number of rows of mix.a1
  mlp:       {kind: "moe", expert: {ff, limit}, router: {experts, identity, top, groups: {count, keep}}}
Tensors:  embed, final.norm, head; per layer that owns tensors l<i>.{norm1, norm1b, norm2, norm2b};
l<i>.mix.{q, k, v, o} and for gla also {g, a1, a2, a2.b, norm}; l<i>.mlp.{router, correction}, l<i>.mlp.e<n>.{gate, up, down};
matrices are [out, in].
"""
from __future__ import annotations

import os
from dataclasses import dataclass, replace

from .checkpoint import make_source, stored_shapes

ARCHITECTURE = "Gerivik"
GLU_ALPHA, GLU_BIAS = 1.702, 1.0        # g sigmoid(alpha g) (u + bias): constants of the design's experts


@dataclass(frozen=True)
class CappedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_base: float
    rot_dims: int                       # leading dimensions of a head that turn with the position
    scale: float
    softcap: float


@dataclass(frozen=True)
class GatedLinearAttention:
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int = 16                # inner size of the decay's two-matrix product


@dataclass(frozen=True)
class RoutedExperts:
    experts: int
    identity: int                       # last outputs of the router: experts that return their input
    top: int
    groups: int
    keep: int
    ff: int
    limit: float

    @property
    def choices(self) -> int:
        return self.experts + self.identity


@dataclass(frozen=True)
class GerivikLayer:
    mixer: CappedAttention | GatedLinearAttention
    mlp: RoutedExperts | None
    weights_of: int | None = None       # layer whose tensors this one uses; None: its own

    @property
    def is_gla(self) -> bool:
        return isinstance(self.mixer, GatedLinearAttention)


@dataclass(frozen=True)
class GerivikConfig:
    name: str
    vocab_size: int
    hidden_size: int
    layers: tuple
    rms_eps: float
    embedding_scale: float
    max_position_embeddings: int = 1 << 20     # no table of positions: a bound for buffers only
    eos_token_ids: tuple = ()

    family = "gerivik"

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def attn_layers(self) -> tuple:
        return tuple(i for i, L in enumerate(self.layers) if not L.is_gla)

    @property
    def gla_layers(self) -> tuple:
        return tuple(i for i, L in enumerate(self.layers) if L.is_gla)

    @property
    def num_attn_layers(self) -> int:
        return len(self.attn_layers)

    @property
    def recurrent(self) -> bool:
        return bool(self.gla_layers)

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        j = self.layers[i].weights_of
        return i if j is None else j

    def validate(self) -> "GerivikConfig":
        for i, L in enumerate(self.layers):
            m, f = L.mixer, L.mlp
            if L.weights_of is not None:
                j = L.weights_of
                if not 0 <= j < len(self.layers) or self.layers[j].weights_of is not None:
                    raise ValueError(f"layer {i}: weights_of must name a layer with tensors of its own, got {j}")
                if replace(L, weights_of=None) != self.layers[j]:
                    raise ValueError(f"layer {i} uses the tensors of layer {j} but is not equal to it")
            if min(m.heads, m.dim, m.vdim) < 1:
                raise ValueError(f"layer {i}: sizes must be positive ({m})")
            if L.is_gla:
                if m.tau <= 0 or m.decay_rank < 1:
                    raise ValueError(f"layer {i}: tau and the decay's rank must be positive ({m})")
            elif m.kv_heads < 1 or m.heads % m.kv_heads or m.rot_dims % 2 or not 0 <= m.rot_dims <= m.dim or m.softcap <= 0:
                raise ValueError(f"layer {i}: bad attention sizes ({m})")
            if f is not None:
                if min(f.experts, f.ff, f.groups, f.keep) < 1 or f.identity < 0 or f.choices % f.groups or f.keep > f.groups:
                    raise ValueError(f"layer {i}: bad expert groups ({f})")
                if not 1 <= f.top <= f.choices // f.groups * f.keep:
                    raise ValueError(f"layer {i}: {f.top} experts cannot be chosen among those of {f.keep} groups")
        return self

    def validate_tp(self, tp: int) -> None:
        if tp > 1:
            raise ValueError("Gerivik runs on one GPU (tp_size = 1)")

    # ---- file format
    @classmethod
    def from_dict(cls, d: dict, name: str = ARCHITECTURE, decay_rank=None) -> "GerivikConfig":
        """`decay_rank`: layer -> rank of its decay product (the tensors carry it, not the file)."""
        if d.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} config: architecture {d.get('architecture')!r}")
        layers = []
        for i, e in enumerate(d["layers"]):
            m, f = e["mixer"], e.get("mlp")
            j = None if e.get("weights_of") is None else int(e["weights_of"])
            if e["type"] == "attention":
                mixer = CappedAttention(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                        rot_base=float(m["rot"]["base"]), rot_dims=int(m["rot"]["dims"]), scale=float(m["scale"]),
                                        softcap=float(m["softcap"]))
            elif e["type"] == "gla":
                mixer = GatedLinearAttention(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), tau=float(m["tau"]))
                rank = (decay_rank or {}).get(i if j is None else j)
                if rank is not None:
                    mixer = replace(mixer, decay_rank=int(rank))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            mlp = None
            if f is not None:
                if f["kind"] != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
                r, g = f["router"], f["router"].get("groups") or {}
                mlp = RoutedExperts(experts=int(r["experts"]), identity=int(r.get("identity") or 0), top=int(r["top"]),
                                    groups=int(g.get("count", 1)), keep=int(g.get("keep", 1)), ff=int(f["expert"]["ff"]),
                                    limit=float(f["expert"]["limit"]))
            layers.append(GerivikLayer(mixer, mlp, j))
        return cls(name=name, vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=tuple(layers),
                   rms_eps=float(d["norm"]["eps"]), embedding_scale=float(d["embedding"]["scale"])).validate()

    def to_dict(self) -> dict:
        layers = []
        for L in self.layers:
            m, f = L.mixer, L.mlp
            if L.is_gla:
                e = {"type": "gla", "mixer": {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "tau": m.tau}}
            else:
                e = {"type": "attention", "mixer": {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim,
                                                    "rot": {"base": m.rot_base, "dims": m.rot_dims}, "scale": m.scale,
                                                    "softcap": m.softcap}}
            e["mlp"] = None if f is None else {
                "kind": "moe", "expert": {"ff": f.ff, "limit": f.limit},
                "router": {"experts": f.experts, "identity": f.identity, "top": f.top, "groups": {"count": f.groups, "keep": f.keep}}}
            if L.weights_of is not None:
                e["weights_of"] = L.weights_of
            layers.append(e)
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "layers": layers,
                "norm": {"eps": self.rms_eps}, "embedding": {"scale": self.embedding_scale}}

    # ---- tensors
    def tensor_shapes(self) -> dict:
        W, V = self.hidden_size, self.vocab_size
        s = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
        for i, L in enumerate(self.layers):
            if L.weights_of is not None:
                continue
            m, f, p = L.mixer, L.mlp, f"l{i}."
            s[p + "norm1"] = s[p + "norm1b"] = (W,)
            s[p + "mix.q"], s[p + "mix.o"] = (m.heads * m.dim, W), (W, m.heads * m.vdim)
            kv = m.heads if L.is_gla else m.kv_heads
            s[p + "mix.k"], s[p + "mix.v"] = (kv * m.dim, W), (kv * m.vdim, W)
            if L.is_gla:
                s[p + "mix.g"], s[p + "mix.norm"] = (m.heads * m.vdim, W), (m.vdim,)
                s[p + "mix.a1"], s[p + "mix.a2"], s[p + "mix.a2.b"] = (m.decay_rank, W), (m.heads * m.dim, m.decay_rank), (m.heads * m.dim,)
            if f is not None:
                s[p + "norm2"] = s[p + "norm2b"] = (W,)
                s[p + "mlp.router"], s[p + "mlp.correction"] = (f.choices, W), (f.choices,)
                for e in range(f.experts):
                    q = f"{p}mlp.e{e}."
                    s[q + "gate"] = s[q + "up"] = (f.ff, W)
                    s[q + "down"] = (W, f.ff)
        return s


def stack(pattern: tuple, repeats: int = 1, shared: int = 0) -> tuple:
    """`repeats` times the layers of `pattern`, each with tensors of its own, then `shared` more rounds on the tensors of
    the first `len(pattern)` layers."""
    own = tuple(pattern) * repeats
    return own + tuple(replace(L, weights_of=i) for _ in range(shared) for i, L in enumerate(pattern))


def _pattern(heads, kv, dim, gla_heads, gla_vdim, mlp, softcap=40.0):
    a = GerivikLayer(CappedAttention(heads=heads, kv_heads=kv, dim=dim, vdim=dim, rot_base=5e5, rot_dims=dim // 4, scale=dim ** -0.5,
                                     softcap=softcap), mlp)
    g = GerivikLayer(GatedLinearAttention(heads=gla_heads, dim=dim, vdim=gla_vdim, tau=12.0), mlp)
    return (g, g, a, g)


TINY = GerivikConfig(
    name="tiny-gerivik", vocab_size=1024, hidden_size=256, rms_eps=1e-6, embedding_scale=16.0, max_position_embeddings=8192,
    layers=stack(_pattern(6, 2, 64, 3, 128, RoutedExperts(experts=14, identity=2, top=3, groups=4, keep=2, ff=128, limit=7.0)), shared=1),
    eos_token_ids=(1023,))

# Layers of the size of a few-billion-parameter models; the benchmark takes as many as it needs.
GERIVIK_2K = GerivikConfig(
    name="gerivik-2k", vocab_size=65536, hidden_size=2048, rms_eps=1e-6, embedding_scale=2048 ** 0.5, max_position_embeddings=32768,
    layers=stack(_pattern(16, 4, 128, 8, 256, RoutedExperts(experts=60, identity=4, top=8, groups=8, keep=4, ff=768, limit=7.0)), repeats=2))
GERIVIK_4K = GerivikConfig(
    name="gerivik-4k", vocab_size=65536, hidden_size=4096, rms_eps=1e-6, embedding_scale=64.0, max_position_embeddings=32768,
    layers=stack(_pattern(32, 8, 128, 16, 256, RoutedExperts(experts=60, identity=4, top=8, groups=8, keep=4, ff=1536, limit=7.0)), repeats=2))

PRESETS = {c.name: c for c in (TINY, GERIVIK_2K, GERIVIK_4K)}


def load_config(model_dir: str, d: dict) -> GerivikConfig:
    rank = {int(n[1:n.index(".")]): s[0] for n, s in stored_shapes(model_dir).items() if n.startswith("l") and n.endswith(".mix.a1")}
    return GerivikConfig.from_dict(d, name=os.path.basename(os.path.normpath(model_dir)) or ARCHITECTURE, decay_rank=rank)


def _random_scale(name: str, shape) -> float:
    """Matrices are scaled by their input size, embeddings too (the configuration scales them up again); the decay's bias
    is N(0, 1)."""
    return 1.0 if name.endswith(".a2.b") else 0.02 if name.endswith(".correction") else shape[-1] ** -0.5


def make_weights(cfg: GerivikConfig, spec: str, model_dir: str | None, device="cpu"):
    return make_source(cfg, spec, model_dir, device, _random_scale)
