"""PyTorch executor of Gerivik on a CPU: paged keys and values, recurrent state slots with snapshots, variable-length
batches, prefix reuse and swapping can be exercised by the engine without a GPU.  (The GPU executor is `gated_b200.py`;
nothing there falls back to this.)
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .gerivik import GLU_ALPHA, GLU_BIAS, GerivikConfig
from .reference_cpu import Batch, rmsnorm, rope_partial
from .weights import fake_quant


class TorchGatedModel:
    def __init__(self, cfg: GerivikConfig, src, *, quant: str = "none", dtype=torch.float32, tp: int = 1, rank: int = 0, comm=None):
        cfg.validate_tp(tp)
        self.cfg, self.dtype, self.tp, self.rank, self.comm = cfg, dtype, tp, rank, comm
        self.vocab_start, self.block_size = 0, 16
        self.w = {n: src.get(n).to(dtype) for n in cfg.tensor_shapes()}
        if quant == "w8a16":
            for n in self.w:
                if n.endswith((".q", ".k", ".v", ".g", ".o", ".a1", ".gate", ".up", ".down")):
                    self.w[n] = fake_quant(self.w[n]).to(dtype)
        self.kv, self.state, self.snapshots = {}, {}, {}

    # ---- cache and state
    def alloc_cache(self, num_blocks: int, block_size: int, num_slots: int):
        self.block_size = block_size
        n = num_blocks * block_size
        for i in self.cfg.attn_layers:
            m = self.cfg.layers[i].mixer
            self.kv[i] = (torch.zeros(n, m.kv_heads, m.dim, dtype=self.dtype), torch.zeros(n, m.kv_heads, m.vdim, dtype=self.dtype))
        for i in self.cfg.gla_layers:
            m = self.cfg.layers[i].mixer
            self.state[i] = torch.zeros(num_slots, m.heads, m.dim, m.vdim)

    def cache_bytes_per_block(self) -> int:
        return sum(self.block_size * c[0].numel() * c.element_size() for kv in self.kv.values() for c in kv)

    def zero_state(self, slot: int):
        for s in self.state.values():
            s[slot].zero_()

    def state_out(self, slot: int):
        return [s[slot].clone() for s in self.state.values()]

    def state_in(self, slot: int, st):
        for s, old in zip(self.state.values(), st):
            s[slot].copy_(old)

    def _rows(self, block_ids: list) -> torch.Tensor:
        bs = self.block_size
        return torch.tensor([b * bs + j for b in block_ids for j in range(bs)], dtype=torch.long)

    def blocks_out(self, block_ids: list):
        rows = self._rows(block_ids)
        return [(k[rows].clone(), v[rows].clone()) for k, v in self.kv.values()]

    def blocks_in(self, block_ids: list, data):
        rows = self._rows(block_ids)
        for (k, v), (dk, dv) in zip(self.kv.values(), data):
            k[rows], v[rows] = dk, dv

    def take_snapshots(self):
        out, self.snapshots = self.snapshots, {}
        return out

    # ---- layers
    def _attention(self, i: int, p: str, h, batch: Batch):
        w, m = self.w, self.cfg.layers[i].mixer
        T, G = h.shape[0], m.kv_heads
        one = torch.ones(m.dim)
        turn = lambda x: rmsnorm(rope_partial(x.float(), batch.positions, m.rot_dims, m.rot_base), one, self.cfg.rms_eps, one_plus=False)
        q = turn((h @ w[p + "q"].t()).view(T, m.heads, m.dim))
        k = turn((h @ w[p + "k"].t()).view(T, G, m.dim)).to(self.dtype)
        v = (h @ w[p + "v"].t()).view(T, G, m.vdim)
        kc, vc = self.kv[i]
        keep = batch.slot_mapping >= 0
        kc[batch.slot_mapping[keep]], vc[batch.slot_mapping[keep]] = k[keep], v[keep]
        out, bs = torch.empty(T, m.heads * m.vdim, dtype=self.dtype), self.block_size
        for s in range(batch.num_seqs):
            t0, t1, end, table = batch.cu_seqlens[s], batch.cu_seqlens[s + 1], batch.context_lens[s], batch.block_tables[s]
            rows = torch.tensor([table[j // bs] * bs + j % bs for j in range(end)], dtype=torch.long)
            qq = q[t0:t1].view(t1 - t0, G, -1, m.dim)
            score = torch.einsum("tgad,jgd->gatj", qq, kc[rows].float()) * m.scale
            score = m.softcap * torch.tanh(score / m.softcap)
            later = batch.positions[t0:t1, None] < torch.arange(end)[None]
            a = torch.softmax(score.masked_fill(later, float("-inf")), dim=-1)
            out[t0:t1] = torch.einsum("gatj,jgv->tgav", a, vc[rows].float()).reshape(t1 - t0, -1).to(self.dtype)
        return out @ w[p + "o"].t()

    def _gla(self, i: int, p: str, h, batch: Batch):
        w, m = self.w, self.cfg.layers[i].mixer
        T, H = h.shape[0], m.heads
        q = (h @ w[p + "q"].t()).float().view(T, H, m.dim) * m.dim ** -0.5
        k = (h @ w[p + "k"].t()).float().view(T, H, m.dim)
        v = (h @ w[p + "v"].t()).float().view(T, H, m.vdim)
        z = (h @ w[p + "a1"].t()).float() @ w[p + "a2"].float().t() + w[p + "a2.b"].float()
        alpha = torch.exp(F.logsigmoid(z) / m.tau).view(T, H, m.dim)
        o = torch.empty(T, H, m.vdim)
        for s in range(batch.num_seqs):
            t0, t1 = batch.cu_seqlens[s], batch.cu_seqlens[s + 1]
            S, first = self.state[i][batch.state_slots[s]], batch.context_lens[s] - (t1 - t0)
            points = set(batch.snapshot_at[s]) if batch.snapshot_at else ()
            for t in range(t0, t1):
                S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
                o[t] = torch.einsum("hdv,hd->hv", S, q[t])
                if first + t - t0 + 1 in points:
                    self.snapshots.setdefault((s, first + t - t0 + 1), []).append(S.clone())
            self.state[i][batch.state_slots[s]] = S
        o = rmsnorm(o, w[p + "norm"], self.cfg.rms_eps, one_plus=False).reshape(T, -1)
        return (o * F.silu((h @ w[p + "g"].t()).float())).to(self.dtype) @ w[p + "o"].t()

    def _experts(self, f, p: str, h):
        w = self.w
        s = torch.softmax(h.float() @ w[p + "router"].float().t(), dim=-1)
        choice = s + w[p + "correction"].float()
        best = choice.view(-1, f.groups, f.choices // f.groups).amax(-1).topk(f.keep, dim=-1).indices
        kept = torch.zeros(h.shape[0], f.groups, dtype=torch.bool).scatter_(1, best, True)
        kept = kept.repeat_interleave(f.choices // f.groups, dim=1)
        ids = choice.masked_fill(~kept, float("-inf")).topk(f.top, dim=-1).indices
        share = torch.zeros_like(s).scatter_(1, ids, s.gather(1, ids))
        out = h.float() * share[:, f.experts:].sum(-1, keepdim=True)
        for e in range(f.experts):
            t = torch.nonzero(share[:, e]).flatten()
            if len(t):
                q = f"{p}e{e}."
                g, u = (h[t] @ w[q + "gate"].t()).clamp(max=f.limit), (h[t] @ w[q + "up"].t()).clamp(-f.limit, f.limit)
                y = (g * torch.sigmoid(GLU_ALPHA * g) * (u + GLU_BIAS)) @ w[q + "down"].t()
                out[t] += share[t, e, None] * y.float()
        return out

    @torch.no_grad()
    def forward(self, batch: Batch) -> torch.Tensor:
        """Normalised hidden states of the last token of every sequence (or of `batch.out_rows`)."""
        c, w = self.cfg, self.w
        norm = lambda x, n: rmsnorm(x, w[n], c.rms_eps, one_plus=False)
        x = w["embed"][batch.input_ids].float() * c.embedding_scale
        self.snapshots = {}
        for i, L in enumerate(c.layers):
            p = f"l{c.owner(i)}."
            mixer = self._gla if L.is_gla else self._attention
            x = x + norm(mixer(i, p + "mix.", norm(x, p + "norm1").to(self.dtype), batch).float(), p + "norm1b")
            if L.mlp is not None:
                x = x + norm(self._experts(L.mlp, p + "mlp.", norm(x, p + "norm2").to(self.dtype)), p + "norm2b")
        rows = batch.out_rows if batch.out_rows is not None else [e - 1 for e in batch.cu_seqlens[1:]]
        return norm(x[rows], "final.norm").to(self.dtype)

    @torch.no_grad()
    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return (hidden @ self.w["head"].t()).float()
