"""Windowed attention over paged keys and values, of the executors on the GPU whose layers have it beside other mixers: the
padding of heads, the buffers and the launches.  A layer object carries sizes, window, scale, slopes, gates (g_col: a column
per head, gate_col: a column per output dimension) and the factor of the output."""
from __future__ import annotations

import torch

from ..ops import functional as F
from ..ops.functional import AttnGeneralParams, AttnParams, ptr
from .paged_state_b200 import PAGE
from .products_b200 import pad64, pad_to
from .runtime_b200 import StepCtx

LOG2E = 1.4426950408889634


def pad_up(n: int, sizes) -> int:
    return next((s for s in sizes if s >= n), pad64(n))


def pad8(n: int) -> int:
    return -(-n // 8) * 8


def head_rows(w: torch.Tensor, H: int, n: int, np_: int) -> torch.Tensor:
    """[H * n, ...] rows of H heads -> [H * np_, ...], each head padded with zero rows."""
    return pad_to(w.reshape(H, n, -1), H, np_, w.numel() // (H * n)).reshape(H * np_, *w.shape[1:])


class AttentionLayers:
    def _attention_sizes(self, L, m):
        sizes = (64, 128, 256) if not self.f32 and max(m.dim, m.vdim) <= 256 else ()
        L.attn, L.heads, L.G, L.dp, L.vp = True, m.heads, m.kv_heads, pad_up(m.dim, sizes), pad_up(m.vdim, sizes)
        if max(L.dp, L.vp) > 1024:
            raise ValueError(f"attention takes heads of at most 1024, got {max(m.dim, m.vdim)}")
        G = m.heads // m.kv_heads                            # query heads of a block: at most 16
        L.rep = G // max(d for d in range(1, 17) if G % d == 0)
        L.k_col, L.v_col = L.heads * L.dp, (L.heads + L.G) * L.dp
        L.window, L.scale, L.slopes, L.g_col, L.gate_col, L.out_scale = m.window, m.scale, None, None, None, 1.0

    def _out_columns(self, w, H: int, n: int, np_: int):
        """Columns of an output matrix for padded heads."""
        return pad_to(w.view(-1, H, n), w.shape[0], H, np_).reshape(w.shape[0], H * np_)

    def _angles(self, base: float, dims: int) -> torch.Tensor:
        return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64).float().to(self.dev)

    def _alloc_attention(self, x: StepCtx, T: int, num_qg: int, nsplit: int, layers: list, new):
        """Query rows, and the partial results of the split attention."""
        if not layers:
            return
        x.q = new(T * max(L.heads * L.dp for L in layers), dtype=self.dtype, device=self.dev)
        if num_qg and not self.f32:
            items = max(num_qg * L.G * L.rep * nsplit * (L.vp if L.vp <= 256 else 0) for L in layers)
            x.o_part = torch.empty(items * 16, dtype=torch.float32, device=self.dev)
            x.ml_part = torch.empty(items // 64 * 32, dtype=torch.float32, device=self.dev)

    def _attention(self, L, x: StepCtx, q, proj, mix):
        """Windowed attention of the step's tokens over the cache pages into the leading columns of mix."""
        kc, vc = self.cache[L.index]
        if x.num_qg:
            general = self.f32 or max(L.dp, L.vp) > 256
            a = AttnGeneralParams() if general else AttnParams()
            a.q, a.kcache, a.vcache, a.block_tables, a.positions = ptr(q), ptr(kc), ptr(vc), ptr(x.block_tables), ptr(x.positions)
            a.qg_seq, a.qg_tok0, a.qg_ntok, a.out, a.status = ptr(x.qg[0]), ptr(x.qg[1]), ptr(x.qg[2]), ptr(mix), self.status
            a.max_blocks, a.num_qg, a.num_blocks, a.ldo = x.max_blocks, x.num_qg, self.num_blocks, mix.stride(0)
            a.window, a.slopes, a.out_scale = L.window, ptr(L.slopes), L.out_scale
            if L.g_col is not None:
                a.head_gate, a.ldg, a.gcol = ptr(proj), proj.stride(0), L.g_col
            if L.gate_col is not None and general:
                a.gate, a.ldg, a.gcol = ptr(proj), proj.stride(0), L.gate_col
            elif L.gate_col is not None:
                a.gate_src, a.ld, a.gate_col, a.gate_stride = ptr(proj), proj.stride(0), L.gate_col, L.vp
            if general:
                a.H, a.G, a.dp, a.vp, a.scale = L.heads, L.G, L.dp, L.vp, L.scale
                F.attn_general(a, self.f32)
            else:
                a.o_part, a.ml_part, a.scale_log2e = ptr(x.o_part), ptr(x.ml_part), L.scale * LOG2E
                # a split takes a page per warp at least
                a.hq, a.hkv, a.rep, a.nsplit = L.heads, L.G, L.rep, max(1, min(x.nsplit, (L.window // PAGE + 2) // 4))
                F.attn_paged(a, L.dp, L.vp)
            self._launches += 1 + (not general)
        if x.tiles is not None:
            F.attn_prefill(q, kc, vc, self.num_blocks, x.block_tables, x.positions, x.tiles,
                           None if L.gate_col is None else proj, mix, hq=L.heads, hkv=L.G, D=L.dp, DV=L.vp, max_blocks=x.max_blocks,
                           ld=0 if L.gate_col is None else proj.stride(0), scale=L.scale, window=L.window, slopes=L.slopes,
                           head_gate=None if L.g_col is None else proj, gcol=L.g_col or 0, out_scale=L.out_scale,
                           gate_col=L.gate_col or 0, gate_stride=L.vp if L.gate_col is not None else 0)
            self._launches += 1
