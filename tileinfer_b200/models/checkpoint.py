"""Weight sources shared by the model families whose checkpoints are a config.json beside safetensors files with the
framework's own tensor names: a reader that checks every shape against the configuration, and seeded random weights."""
from __future__ import annotations

import hashlib
import os

import torch


class _Files:
    """The safetensors files of a folder: tensor name -> open file."""

    def __init__(self, model_dir: str):
        from safetensors import safe_open
        self.where = {}
        for fn in sorted(f for f in os.listdir(model_dir) if f.endswith(".safetensors")):
            h = safe_open(os.path.join(model_dir, fn), "pt")
            for k in h.keys():
                self.where[k] = h

    def shape(self, name: str) -> tuple:
        return tuple(self.where[name].get_slice(name).get_shape())


def stored_shapes(model_dir: str) -> dict:
    """Tensor name -> shape of every tensor in the folder (empty when it holds none)."""
    f = _Files(model_dir)
    return {k: f.shape(k) for k in f.where}


class CheckpointWeights:
    """Reads a checkpoint folder tensor by tensor (model.safetensors, or shards with an index)."""

    def __init__(self, cfg, model_dir: str, device="cpu"):
        self.cfg, self.device = cfg, torch.device(device)
        self._files = _Files(model_dir)
        for name, shape in cfg.tensor_shapes().items():
            if name not in self._files.where:
                raise ValueError(f"{model_dir}: no tensor {name}")
            have = self._files.shape(name)
            if have != tuple(shape):
                raise ValueError(f"{model_dir}: {name} has shape {have}, the configuration says {tuple(shape)}")

    def get(self, name: str) -> torch.Tensor:
        """Full tensor in fp32 on `self.device`."""
        return self._files.where[name].get_tensor(name).to(self.device).float()


class RandomWeights:
    """Deterministic weights of the architecture: every tensor has its own generator stream.  Norm weights are 1
    (those that `zero_norm(name)` says are stored around zero: 0); the N(0, 1) draws of the others go through
    `scale_of(name, shape)` and are rounded to bf16."""

    def __init__(self, cfg, seed: int, device, scale_of, zero_norm=None):
        self.cfg, self.seed, self.device, self._scale_of = cfg, seed, torch.device(device), scale_of
        self._zero_norm = zero_norm or (lambda name: False)
        self._shapes = cfg.tensor_shapes()

    def get(self, name: str) -> torch.Tensor:
        shape = self._shapes[name]
        if "norm" in name.rsplit(".", 1)[-1]:
            return torch.full(shape, 0.0 if self._zero_norm(name) else 1.0, dtype=torch.float32, device=self.device)
        # small tensors come from the CPU generator so that CPU and GPU runs see the same weights
        numel = 1
        for n in shape:
            numel *= n
        dev = torch.device("cpu") if numel <= 1 << 24 else self.device
        g = torch.Generator(device=dev)
        g.manual_seed(int.from_bytes(hashlib.sha256(f"{self.seed}:{name}".encode()).digest()[:7], "little"))
        w = torch.empty(shape, dtype=torch.float32, device=dev).normal_(0.0, 1.0, generator=g) * self._scale_of(name, shape)
        return w.to(torch.bfloat16).float().to(self.device)


def make_source(cfg, spec: str, model_dir, device, scale_of, zero_norm=None):
    """`spec` is "random:<seed>" or "hf" (a checkpoint folder)."""
    if spec.startswith("random"):
        return RandomWeights(cfg, int(spec.split(":", 1)[1]) if ":" in spec else 0, device, scale_of, zero_norm)
    if spec == "hf":
        return CheckpointWeights(cfg, model_dir, device)
    raise ValueError(f"unknown weights spec {spec!r}")
