"""Weights in kernel layout for designs with an fp32 residual: plain products and products of token groups with experts, in
bf16, int8 or 32-bit, behind one call."""
from __future__ import annotations

import torch

from ..ops import functional as F
from ..ops.functional import LinearW


def pad64(n: int) -> int:
    return -(-n // 64) * 64


def pad_to(t: torch.Tensor, *shape) -> torch.Tensor:
    """`t` in the corner of a zero tensor of the given shape."""
    out = t.new_zeros(shape)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


class Product:
    """y = x W^T with the epilogues of a fp32-residual model, in one of three weight formats."""

    def __init__(self, w: torch.Tensor, quant: str, dev):
        self.N, self.K = w.shape
        self.f32 = quant == "fp32"
        self.w = w.to(dev, torch.float32).contiguous() if self.f32 else LinearW(w, quant == "w8a16", dev)

    def nbytes(self) -> int:
        return self.w.numel() * 4 if self.f32 else self.w.nbytes()

    def __call__(self, x, out, epi, ex=None) -> int:
        """Returns the number of kernels launched."""
        if self.f32:
            F.gemm_f32(self.w, x, out=out, epi=F.GEPI_F32 if epi == F.GEPI_STORE else epi, ex=ex)
            return 1
        if self.w.wt == F.W_INT8:
            F.gemm_w8a16(self.w, F.quant_rows(x), out=out, epi=epi, ex=ex)
            return 2
        F.gemm_bf16(self.w, x, out=out, epi=epi, ex=ex)
        return 1


class GroupedProduct:
    """y[r] = x[r] W_e^T for rows grouped by expert; `weights`: the E matrices [N, K], N a multiple of 8."""

    def __init__(self, weights, quant: str, dev):
        self.E, (self.N, self.K) = len(weights), weights[0].shape
        self.f32 = quant == "fp32"
        self.w = torch.stack([w.to(dev, torch.float32) for w in weights]) if self.f32 else LinearW(torch.cat(weights), quant == "w8a16", dev)

    def nbytes(self) -> int:
        return self.w.numel() * 4 if self.f32 else self.w.nbytes()

    def __call__(self, x, groups, out, epi, ex=None) -> int:
        """Returns the number of kernels launched."""
        if self.f32:
            F.gemm_f32(self.w, x, out=out, epi=F.GEPI_F32 if epi == F.GEPI_STORE else epi, ex=ex, groups=groups)
            return 1
        if self.w.wt == F.W_INT8:
            F.gemm_grouped(self.w, self.E, F.quant_rows(x), groups, out=out, epi=epi, ex=ex)
            return 2
        F.gemm_grouped(self.w, self.E, x, groups, out=out, epi=epi, ex=ex)
        return 1
