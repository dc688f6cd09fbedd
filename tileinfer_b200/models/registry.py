"""Model families: how a configuration is recognised, where its weights come from and which executors run it.

The engine knows a model only through its configuration object (`family` names the entry here) and through the executor
interface (`alloc_cache`, `forward`, `logits`, `forward_and_sample`, ...).  A new design adds one entry.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable


@dataclass(frozen=True)
class Family:
    name: str
    presets: Callable                   # () -> {preset name: configuration}
    architecture: str | None            # "architecture" of its config.json; None: a HuggingFace configuration
    load_config: Callable               # (model_dir, config.json dict) -> configuration
    make_weights: Callable              # (configuration, spec, model_dir, device) -> weight source
    executor: Callable                  # (device) -> executor class
    quantizations: tuple                # accepted Config.quantization values


def _hybrid() -> Family:
    from .config import PRESETS, from_hf_config
    from .weights import make_weight_source

    def load(model_dir, _):
        from transformers import AutoConfig
        return from_hf_config(AutoConfig.from_pretrained(model_dir, trust_remote_code=False))

    def executor(device):
        if device == "cuda":
            from .hybrid_b200 import B200HybridModel
            return B200HybridModel
        from .reference_cpu import TorchHybridModel
        return TorchHybridModel

    return Family("hybrid", lambda: PRESETS, None, load, make_weight_source, executor, ("w8a16", "bf16"))


def _kabadra() -> Family:
    from . import kabadra as k

    def executor(device):
        if device == "cuda":
            from .latent_b200 import B200LatentModel
            return B200LatentModel
        from .latent_cpu import TorchLatentModel
        return TorchLatentModel

    return Family("kabadra", lambda: k.PRESETS, k.ARCHITECTURE, k.load_config, k.make_weights, executor, ("w8a16", "bf16", "fp32"))


def _gerivik() -> Family:
    from . import gerivik as g

    def executor(device):
        if device == "cuda":
            from .gated_b200 import B200GatedModel
            return B200GatedModel
        from .gated_cpu import TorchGatedModel
        return TorchGatedModel

    return Family("gerivik", lambda: g.PRESETS, g.ARCHITECTURE, g.load_config, g.make_weights, executor, ("w8a16", "bf16", "fp32"))


def _nogidra() -> Family:
    from . import nogidra as n

    def executor(device):
        if device == "cuda":
            from .mixed_b200 import B200MixedModel
            return B200MixedModel
        from .mixed_cpu import TorchMixedModel
        return TorchMixedModel

    return Family("nogidra", lambda: n.PRESETS, n.ARCHITECTURE, n.load_config, n.make_weights, executor, ("w8a16", "bf16", "fp32"))


def _luvapel() -> Family:
    from . import luvapel as v

    def executor(device):
        if device == "cuda":
            from .delta_b200 import B200DeltaModel
            return B200DeltaModel
        from .delta_cpu import TorchDeltaModel
        return TorchDeltaModel

    return Family("luvapel", lambda: v.PRESETS, v.ARCHITECTURE, v.load_config, v.make_weights, executor, ("w8a16", "bf16", "fp32"))


_MAKERS = {"hybrid": _hybrid, "kabadra": _kabadra, "gerivik": _gerivik, "nogidra": _nogidra, "luvapel": _luvapel}


def family(name: str) -> Family:
    return _MAKERS[name]()


def families() -> list:
    return [f() for f in _MAKERS.values()]


def all_presets() -> dict:
    return {n: c for f in families() for n, c in f.presets().items()}


def is_preset(model: str) -> bool:
    return model.startswith("preset:") or model in all_presets()


def get_preset(model: str):
    key = model.split(":", 1)[1] if model.startswith("preset:") else model
    presets = all_presets()
    if key not in presets:
        raise KeyError(f"unknown model preset {model!r}; known: {sorted(presets)}")
    return presets[key]


def config_from_dir(model_dir: str):
    """Configuration of a local model folder; the family is chosen by "architecture" in its config.json."""
    d = {}
    path = os.path.join(model_dir, "config.json")
    if os.path.exists(path):
        with open(path) as f:
            d = json.load(f)
    arch = d.get("architecture")
    for fam in families():
        if fam.architecture == arch:
            return fam.load_config(model_dir, d)
    raise ValueError(f"{model_dir}: unknown architecture {arch!r}")
