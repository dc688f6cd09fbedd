"""PyTorch executor of Kabadra on a CPU: the paged cache of latents, variable-length batches, prefix reuse and swapping
can be exercised by the engine without a GPU.  (The GPU executor is `latent_b200.py`; nothing there falls back to this.)
"""
from __future__ import annotations

import torch

from .kabadra import GLU_ALPHA, GLU_BIAS, KabadraConfig
from .reference_cpu import Batch, rmsnorm
from .weights import fake_quant


class TorchLatentModel:
    def __init__(self, cfg: KabadraConfig, src, *, quant: str = "none", dtype=torch.float32, tp: int = 1, rank: int = 0, comm=None):
        cfg.validate_tp(tp)
        self.cfg, self.dtype, self.tp, self.rank, self.comm = cfg, dtype, tp, rank, comm
        self.vocab_start, self.block_size = 0, 16
        self.w = {n: src.get(n).to(dtype) for n in cfg.tensor_shapes()}
        if quant == "w8a16":
            for n in self.w:
                if n.endswith((".q", ".dkv", ".g", ".o", ".gate", ".up", ".down")):
                    self.w[n] = fake_quant(self.w[n]).to(dtype)
        self.cache = {}
        self.snapshots = {}

    # ---- cache
    def alloc_cache(self, num_blocks: int, block_size: int, num_slots: int):
        self.block_size = block_size
        self.cache = {i: torch.zeros(num_blocks * block_size, self.cfg.layers[i].mixer.kv_rank, dtype=self.dtype)
                      for i in self.cfg.latent_owners}

    def cache_bytes_per_block(self) -> int:
        return sum(self.block_size * c.shape[1] * c.element_size() for c in self.cache.values())

    def zero_state(self, slot: int):
        pass                                   # no recurrent state: the cache blocks are all a sequence has

    def state_out(self, slot: int):
        return None

    def state_in(self, slot: int, st):
        pass

    def _rows(self, block_ids: list) -> torch.Tensor:
        bs = self.block_size
        return torch.tensor([b * bs + j for b in block_ids for j in range(bs)], dtype=torch.long)

    def blocks_out(self, block_ids: list):
        rows = self._rows(block_ids)
        return {i: c[rows].clone() for i, c in self.cache.items()}

    def blocks_in(self, block_ids: list, data):
        rows = self._rows(block_ids)
        for i, c in self.cache.items():
            c[rows] = data[i]

    def take_snapshots(self):
        return {}

    # ---- layers
    def _mixer(self, i: int, h, batch: Batch):
        w, m, p = self.w, self.cfg.layers[i].mixer, f"l{i}.mix."
        cache = self.cache[self.cfg.latent_layer(i)]
        if m.kv_from is None:
            c = rmsnorm(h @ w[p + "dkv"].t(), w[p + "dkv.norm"], self.cfg.rms_eps, one_plus=False).to(self.dtype)
            keep = batch.slot_mapping >= 0
            cache[batch.slot_mapping[keep]] = c[keep]
        q = (h @ w[p + "q"].t()).view(-1, m.heads, m.dim)
        gate = torch.sigmoid((h @ w[p + "g"].t()).float())
        uk, uv = w[p + "uk"].view(m.heads, m.dim, -1), w[p + "uv"].view(m.heads, m.vdim, -1)
        sink = w[p + "sink"].float()
        out = torch.empty(h.shape[0], m.heads, m.vdim, dtype=self.dtype)
        bs = self.block_size
        for s in range(batch.num_seqs):
            t0, t1 = batch.cu_seqlens[s], batch.cu_seqlens[s + 1]
            end, table = batch.context_lens[s], batch.block_tables[s]
            lo = max(0, end - (t1 - t0) - m.window + 1)           # first position any of these tokens sees
            rows = torch.tensor([table[j // bs] * bs + j % bs for j in range(lo, end)], dtype=torch.long)
            c = cache[rows].float()
            qa = torch.einsum("thd,hdr->thr", q[t0:t1].float(), uk.float())
            score = torch.einsum("thr,jr->htj", qa, c) * m.scale
            dist = batch.positions[t0:t1, None] - torch.arange(lo, end)[None]
            score = score.masked_fill(((dist < 0) | (dist >= m.window))[None], float("-inf"))
            full = torch.cat([score, sink[:, None, None].expand(-1, t1 - t0, 1)], dim=-1)
            a = torch.softmax(full, dim=-1)[..., :-1]
            o = torch.einsum("htj,jr->thr", a, c)
            out[t0:t1] = (torch.einsum("thr,hvr->thv", o, uv.float()) * gate[t0:t1, :, None]).to(self.dtype)
        return out.flatten(1) @ w[p + "o"].t()

    def _mlp(self, i: int, h):
        w, p, lim = self.w, f"l{i}.mlp.", self.cfg.layers[i].mlp.limit
        g, u = (h @ w[p + "gate"].t()).clamp(max=lim), (h @ w[p + "up"].t()).clamp(-lim, lim)
        return (g * torch.sigmoid(GLU_ALPHA * g) * (u + GLU_BIAS)) @ w[p + "down"].t()

    @torch.no_grad()
    def forward(self, batch: Batch) -> torch.Tensor:
        """Normalised hidden states of the last token of every sequence (or of `batch.out_rows`)."""
        c, w = self.cfg, self.w
        x = rmsnorm(w["embed"][batch.input_ids] + w["pos"][batch.positions], w["embed.norm"], c.rms_eps, one_plus=False)
        for i, L in enumerate(c.layers):
            h = rmsnorm(x, w[f"l{i}.norm1"], c.rms_eps, one_plus=False).to(self.dtype)
            y = self._mixer(i, h, batch)
            if L.mlp is not None:
                y = y + self._mlp(i, h)
            x = x + y.float()
        rows = batch.out_rows if batch.out_rows is not None else [e - 1 for e in batch.cu_seqlens[1:]]
        return rmsnorm(x[rows], w["final.norm"], c.rms_eps, one_plus=False).to(self.dtype)

    @torch.no_grad()
    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return (hidden @ self.w["head"].t()).float() * self.cfg.logit_scale
