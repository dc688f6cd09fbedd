"""Short causal convolutions over time in front of a mixer, of the executors on the GPU: parameters and the stored form (with
silu).  A layer object carries the filters [taps, channels], the first channel's column and the number of channels."""
from __future__ import annotations

from ..ops import functional as F
from ..ops.functional import ConvParams, ptr
from .runtime_b200 import StepCtx


class ConvLayers:
    def _conv_params(self, L, x: StepCtx, proj) -> ConvParams:
        p = ConvParams()
        p.proj, p.w, p.bias, p.state, p.slots = ptr(proj), ptr(L.conv_w), ptr(L.conv_b), ptr(self.state[L.index, "conv"]), ptr(x.slots)
        p.T, p.S, p.ld, p.col, p.C, p.taps = x.T, x.S, proj.stride(0), L.conv_col, L.C, L.taps
        if x.cu is not None:
            p.cu, p.tiles, p.num_tiles = ptr(x.cu), ptr(x.conv_tiles), x.conv_tiles.shape[1]
        if x.snaps:
            p.snap_rel, p.snap_idx, p.snap, p.num_snap = ptr(x.snap_rel), ptr(x.snap_idx), ptr(x.snap_state[L.index, "conv"]), x.num_snap
        return p

    def _conv_inputs(self, L, x: StepCtx, proj):
        """The channels after convolution and silu."""
        xbc = x.xbc[:x.T * L.C].view(x.T, L.C)
        p = self._conv_params(L, x, proj)
        p.out, p.ldo, p.silu = ptr(xbc), L.C, 1
        F.conv(p, self.f32)
        self._launches += 1 + (x.cu is not None and L.taps > 1)
        return xbc
