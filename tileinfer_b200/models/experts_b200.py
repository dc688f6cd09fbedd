"""Mixture-of-experts feed-forwards of the executors with an fp32 residual: weights, work buffers and the launches between
the mixer's output and the experts' rows.  A layer's sizes are in `L.moe` (experts, identity, top, groups, keep, ff); its
scores are corrected when there is `L.correction`, else the weights are a softmax over the chosen logits."""
from __future__ import annotations

import torch

from ..ops import functional as F
from .products_b200 import GroupedProduct, Product, pad64, pad_to
from .runtime_b200 import StepCtx


class ExpertLayers:
    FEW_TOKENS = 128                 # up to this many tokens the norm kernel routes the rows it makes

    def _build_experts(self, L, f, p: str, get, glu: tuple, correction=None):
        """`p`: prefix of the tensors; `glu`: (limit, alpha, bias) of the gated unit."""
        dev, Wp = self.dev, self.Wp
        if f.choices > 1024:
            raise ValueError(f"the router takes at most 1024 experts, got {f.choices}")
        L.moe, L.ff, L.glu, L.correction = f, pad64(f.ff), glu, correction
        router = pad_to(get(p + "router"), f.choices, Wp)
        L.router, L.router_rows = Product(router, "fp32" if self.f32 else "bf16", dev), router.to(self.dtype).contiguous()
        up, down = [], []
        for e in range(f.experts):
            g, u = (pad_to(get(f"{p}e{e}.{n}"), L.ff, Wp) for n in ("gate", "up"))
            up.append(torch.stack([g, u], dim=1).reshape(2 * L.ff, Wp).to(torch.float32 if self.quant != "bf16" else torch.bfloat16))
            down.append(pad_to(get(f"{p}e{e}.down"), Wp, L.ff).to(up[-1].dtype))
        L.w_up = GroupedProduct(up, self.quant, dev)
        del up
        L.w_down = GroupedProduct(down, self.quant, dev)

    def _expert_bytes(self, L, tokens: int) -> int:
        """Bytes of weights a decode step of `tokens` tokens streams (at most `top` experts per token)."""
        share = min(1.0, tokens * L.moe.top / L.moe.choices)
        return L.router.nbytes() + int((L.w_up.nbytes() + L.w_down.nbytes()) * share)

    def _alloc_experts(self, x: StepCtx, T: int, layers: list, new):
        x.groups = {}
        if not layers:
            return
        few = T <= self.FEW_TOKENS and self.Wp <= F.NORM_ROUTE_MAX_WIDTH
        for L in layers:
            key = (L.moe.experts, L.moe.choices, L.moe.top)
            if key not in x.groups:
                fixed = few and L.moe.experts * T * self.Wp <= 1 << 26
                x.groups[key] = F.TokenGroups(T, *key, self.counters, self.f32, self.dev, fixed)
        rows = max(g.rows for g in x.groups.values())
        x.logits = new(T * max(-(-L.moe.choices // 8) * 8 for L in layers), dtype=torch.float32, device=self.dev)
        x.xs = new(rows * self.Wp, dtype=self.dtype, device=self.dev)      # token rows by expert, then the experts' outputs
        x.act = new(rows * max(L.ff for L in layers), dtype=self.dtype, device=self.dev)

    def _norm_and_route(self, L, x: StepCtx, y, norm_out):
        """Adds y (through the norm `norm_out`; either may be None) to the residual; the experts' input x.h, its routing and
        its rows by expert."""
        f, T, c, Wp = L.moe, x.T, self.cfg, self.Wp
        g = x.groups[(f.experts, f.choices, f.top)]
        xs = x.xs[:g.rows * Wp].view(g.rows, Wp)
        if g.row_stride:
            F.moe_norm_route(y, x.x, norm_out, x.h, L.norm2, self.W, c.rms_eps, g, L.router_rows, L.correction, f.groups, f.keep, xs,
                             valid=x.slot_mapping)
            self._launches += 1
        else:
            F.resid_norm(y, x.x, norm_out, x.h, L.norm2, self.W, c.rms_eps)
            n = -(-f.choices // 8) * 8
            logits = x.logits[:T * n].view(T, n)
            self._launches += 3 + L.router(x.h, logits, F.GEPI_F32)
            F.moe_route(g, logits, L.correction, f.groups, f.keep, valid=x.slot_mapping)
            F.moe_permute(g, x.h, xs)
        return g, xs

    def _experts(self, L, x: StepCtx, g, xs):
        """The experts' outputs, in the place of their rows."""
        act = x.act[:g.rows * L.ff].view(g.rows, L.ff)
        ex = F.gemm_epilogue(out2=act, n_split=0, glu=L.glu)
        self._launches += L.w_up(xs, g, None, F.GEPI_SPLIT_GLU, ex) + L.w_down(act, g, xs, F.GEPI_STORE)
