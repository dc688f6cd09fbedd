"""PyTorch executor of Nogidra on a CPU: pages of keys, values and latents, recurrent states and convolution tails in slots
with snapshots, variable-length batches, prefix reuse and swapping can be exercised by the engine without a GPU.  (The GPU
executor is `mixed_b200.py`; nothing there falls back to this.)
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .nogidra import ConvAttention, DenseGlu, NogidraConfig, ParallelMixer, RotaryLatent
from .reference_cpu import Batch, rmsnorm, rope_partial
from .weights import fake_quant


def turn_pairs(x, positions, dims, base):
    """Neighbouring dimensions (2i, 2i + 1) of x [T, heads, dim] turn together."""
    inv = base ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims)
    a = positions[:, None, None].float() * inv.float()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()], -1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], -1)


class TorchMixedModel:
    QUANTISED = (".q", ".k", ".v", ".g", ".o", ".dkv", ".in", ".gate", ".up", ".down")

    def __init__(self, cfg: NogidraConfig, src, *, quant: str = "none", dtype=torch.float32, tp: int = 1, rank: int = 0, comm=None):
        cfg.validate_tp(tp)
        self.cfg, self.dtype, self.tp, self.rank, self.comm = cfg, dtype, tp, rank, comm
        self.vocab_start, self.block_size = 0, 16
        self.w = {n: src.get(n).to(dtype) for n in cfg.tensor_shapes()}
        if quant == "w8a16":
            for n in self.w:
                if n.endswith(self.QUANTISED):
                    self.w[n] = fake_quant(self.w[n]).to(dtype)
        self.pages, self.state, self.snapshots = {}, {}, {}

    # ---- cache and state
    def alloc_cache(self, num_blocks: int, block_size: int, num_slots: int):
        self.block_size = block_size
        n = num_blocks * block_size
        for i, L in enumerate(self.cfg.layers):
            m = L.mixer
            if isinstance(m, RotaryLatent):
                self.pages[i] = (torch.zeros(n, m.kv_rank + m.rot_dim, dtype=self.dtype),)
                continue
            a = m.left if isinstance(m, ParallelMixer) else m
            self.pages[i] = (torch.zeros(n, a.kv_heads, a.dim, dtype=self.dtype), torch.zeros(n, a.kv_heads, a.vdim, dtype=self.dtype))
            if isinstance(m, ParallelMixer):
                r = m.right
                self.state[i, "ssm"] = torch.zeros(num_slots, r.heads, r.state, r.vdim)
                self.state[i, "conv"] = torch.zeros(num_slots, r.taps - 1, r.conv_channels, dtype=self.dtype)
            else:
                rows = m.heads * m.dim + m.kv_heads * (m.dim + m.vdim)
                self.state[i, "conv"] = torch.zeros(num_slots, m.taps - 1, rows, dtype=self.dtype)

    def cache_bytes_per_block(self) -> int:
        return sum(self.block_size * c[0].numel() * c.element_size() for p in self.pages.values() for c in p)

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
        return [c[rows].clone() for p in self.pages.values() for c in p]

    def blocks_in(self, block_ids: list, data):
        rows = self._rows(block_ids)
        for c, d in zip((c for p in self.pages.values() for c in p), data):
            c[rows] = d

    def take_snapshots(self):
        out, self.snapshots = self.snapshots, {}
        return out

    # ---- parts
    def _linear(self, h, name: str):
        y = h @ self.w[name].t()
        return y + self.w[name + ".b"] if name + ".b" in self.w else y

    def _sequences(self, batch: Batch):
        """(sequence, first row, one past its last, first position, positions to snapshot after) of every sequence."""
        for s in range(batch.num_seqs):
            t0, t1 = batch.cu_seqlens[s], batch.cu_seqlens[s + 1]
            yield s, t0, t1, batch.context_lens[s] - (t1 - t0), (batch.snapshot_at[s] if batch.snapshot_at else ())

    def _snapshot(self, s: int, at: int, key, value):
        self.snapshots.setdefault((s, at), {})[key] = value.clone()

    def _conv(self, i: int, u, w, batch: Batch):
        """Causal convolution over time of u [T, channels] with w [channels, taps]; the tails are carried in the state."""
        taps, y, key = w.shape[1], torch.empty(u.shape, dtype=torch.float32), (i, "conv")
        for s, t0, t1, first, points in self._sequences(batch):
            slot = batch.state_slots[s]
            past = torch.cat([self.state[key][slot], u[t0:t1].to(self.dtype)])
            y[t0:t1] = sum(w[:, j].float() * past[j:j + t1 - t0].float() for j in range(taps))
            for a in points:
                self._snapshot(s, a, key, past[a - first:a - first + taps - 1])
            self.state[key][slot] = past[len(past) - (taps - 1):]
        return y

    def _store(self, page, rows, batch: Batch):
        keep = batch.slot_mapping >= 0
        page[batch.slot_mapping[keep]] = rows[keep].to(self.dtype)

    def _seen(self, batch: Batch, window: int):
        """Per sequence: its rows, the cache rows in reach, distances [T, keys] and which of them are out of the window."""
        bs = self.block_size
        for s, t0, t1, first, _ in self._sequences(batch):
            lo, table = max(0, first - window + 1), batch.block_tables[s]
            rows = torch.tensor([table[j // bs] * bs + j % bs for j in range(lo, batch.context_lens[s])], dtype=torch.long)
            dist = batch.positions[t0:t1, None] - torch.arange(lo, batch.context_lens[s])[None]
            yield t0, t1, rows, dist, (dist < 0) | (dist >= window)

    def _attend(self, i: int, m, q, batch: Batch, slopes=None):
        """q [T, heads, dim] (fp32) against the layer's pages -> [T, heads, vdim] in fp32."""
        G, (kc, vc) = m.kv_heads, self.pages[i]
        out = torch.empty(q.shape[0], m.heads, m.vdim)
        for t0, t1, rows, dist, hidden in self._seen(batch, m.window):
            score = torch.einsum("tgad,jgd->gatj", q[t0:t1].view(t1 - t0, G, -1, m.dim), kc[rows].float()) * m.scale
            if slopes is not None:
                score = score - torch.tensor(slopes).view(G, -1, 1, 1) * dist.float()
            a = torch.softmax(score.masked_fill(hidden, float("-inf")), dim=-1)
            out[t0:t1] = torch.einsum("gatj,jgv->tgav", a, vc[rows].float()).reshape(t1 - t0, m.heads, m.vdim)
        return out

    # ---- mixers
    def _conv_attention(self, i: int, m: ConvAttention, p: str, h, batch: Batch):
        w, T = self.w, h.shape[0]
        u = torch.cat([h @ w[p + n].t() for n in "qkv"], 1)
        y = self._conv(i, u, torch.cat([w[f"{p}{n}.conv"] for n in "qkv"]), batch)
        q, k, v = y.split([m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim], 1)
        temp = 1.0 + m.temp_coef * torch.log(((batch.positions + 1) // m.temp_every + 1).float())
        self._store(self.pages[i][0], k.view(T, m.kv_heads, m.dim), batch)
        self._store(self.pages[i][1], v.view(T, m.kv_heads, m.vdim), batch)
        o = self._attend(i, m, q.view(T, m.heads, m.dim) * temp[:, None, None], batch, m.slopes())
        o = o * torch.sigmoid((h @ w[p + "g"].t()).float())[..., None]
        return o.reshape(T, -1).to(self.dtype) @ w[p + "o"].t()

    def _latent(self, i: int, m: RotaryLatent, p: str, h, batch: Batch):
        w, T, H, R = self.w, h.shape[0], m.heads, m.kv_rank
        turn = lambda x: rope_partial(x.float(), batch.positions, m.rot_dim, m.rot_base) if m.rot_dim else x.float()
        q = (h @ w[p + "q"].t()).view(T, H, -1)
        down = h @ w[p + "dkv"].t()
        c = rmsnorm(down[:, :R], w[p + "dkv.norm"], self.cfg.rms_eps, one_plus=False)
        self._store(self.pages[i][0], torch.cat([c.float(), turn(down[:, None, R:])[:, 0]], 1), batch)
        uk, uv = w[p + "uk"].view(H, m.dim, R).float(), w[p + "uv"].view(H, m.vdim, R).float()
        q = torch.cat([torch.einsum("thd,hdr->thr", q[..., :m.dim].float(), uk), turn(q[..., m.dim:])], -1)
        out = torch.empty(T, H, m.vdim, dtype=self.dtype)
        for t0, t1, rows, _, hidden in self._seen(batch, m.window):
            c = self.pages[i][0][rows].float()
            a = torch.softmax((torch.einsum("thr,jr->htj", q[t0:t1], c) * m.scale).masked_fill(hidden, float("-inf")), dim=-1)
            out[t0:t1] = torch.einsum("thr,hvr->thv", torch.einsum("htj,jr->thr", a, c[:, :R]), uv).to(self.dtype)
        return out.flatten(1) @ w[p + "o"].t()

    def _parallel(self, i: int, m: ParallelMixer, p: str, h, batch: Batch):
        return m.left_scale * self._normed(i, m.left, p + "left.", h, batch) + m.right_scale * self._state_space(i, m.right, p + "right.", h, batch)

    def _normed(self, i: int, m, p: str, h, batch: Batch):
        T, eps = h.shape[0], self.cfg.rms_eps
        part = lambda n, heads: turn_pairs(rmsnorm(self._linear(h, p + n).float(), self.w[f"{p}{n}.norm"], eps, one_plus=False)
                                            .view(T, heads, m.dim), batch.positions, m.rot_dims, m.rot_base)
        self._store(self.pages[i][0], part("k", m.kv_heads), batch)
        self._store(self.pages[i][1], self._linear(h, p + "v").view(T, m.kv_heads, m.vdim), batch)
        return self._attend(i, m, part("q", m.heads), batch).reshape(T, -1).to(self.dtype) @ self.w[p + "o"].t()

    def _state_space(self, i: int, m, p: str, h, batch: Batch):
        w, T = self.w, h.shape[0]
        z, u, dt = (h @ w[p + "in"].t()).split([m.inner, m.conv_channels, m.heads], 1)
        u = F.silu(self._conv(i, u, w[p + "conv"], batch) + w[p + "conv.b"].float()).to(self.dtype).float()
        x, B, C = u.split([m.inner, m.groups * m.state, m.groups * m.state], 1)
        spread = lambda t: t.view(T, m.groups, m.state).repeat_interleave(m.heads // m.groups, 1)
        x, B, C = x.view(T, m.heads, m.vdim), spread(B), spread(C)
        dt = F.softplus(dt.float() + w[p + "dt_bias"].float(), threshold=1e9)
        decay = torch.exp(-torch.exp(w[p + "A_log"].float()) * dt)
        y = torch.empty(T, m.heads, m.vdim)
        for s, t0, t1, first, points in self._sequences(batch):
            S = self.state[i, "ssm"][batch.state_slots[s]]
            for t in range(t0, t1):
                S = decay[t][:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None, :]
                y[t] = torch.einsum("hnv,hn->hv", S, C[t])
                if first + t - t0 + 1 in points:
                    self._snapshot(s, first + t - t0 + 1, (i, "ssm"), S)
            self.state[i, "ssm"][batch.state_slots[s]] = S
        y = (y + w[p + "D"].float()[:, None] * x).reshape(T, -1) * F.silu(z.float())
        one = torch.ones(m.inner // m.norm_groups)
        y = rmsnorm(y.view(T, m.norm_groups, -1), one, self.cfg.rms_eps, one_plus=False).reshape(T, -1) * w[p + "norm"].float()
        return y.to(self.dtype) @ w[p + "o"].t()

    # ---- feed-forward
    def _unit(self, h, p: str):
        return self._linear(F.silu(self._linear(h, p + "gate")) * self._linear(h, p + "up"), p + "down")

    def _mlp(self, f, p: str, h):
        if isinstance(f, DenseGlu):
            return self._unit(h, p)
        z, ids = (h.float() @ self.w[p + "router"].float().t()).topk(f.top, dim=-1)
        share = torch.zeros(h.shape[0], f.experts).scatter_(1, ids, torch.softmax(z, -1))
        out = torch.zeros(h.shape, dtype=torch.float32)
        for e in range(f.experts):
            t = torch.nonzero(share[:, e]).flatten()
            if len(t):
                out[t] += share[t, e, None] * self._unit(h[t], f"{p}e{e}.").float()
        return out

    @torch.no_grad()
    def forward(self, batch: Batch) -> torch.Tensor:
        """Normalised hidden states of the last token of every sequence (or of `batch.out_rows`)."""
        c, w = self.cfg, self.w
        norm = lambda x, n: rmsnorm(x, w[n], c.rms_eps).to(self.dtype)
        mixers = {ConvAttention: self._conv_attention, RotaryLatent: self._latent, ParallelMixer: self._parallel}
        x = w["embed"][batch.input_ids].float()
        self.snapshots = {}
        for i, L in enumerate(c.layers):
            x = x + mixers[type(L.mixer)](i, L.mixer, f"l{i}.mix.", norm(x, f"l{i}.norm1"), batch).float()
            if L.mlp is not None:
                x = x + self._mlp(L.mlp, f"l{i}.mlp.", norm(x, f"l{i}.norm2")).float()
        self.snapshots = {k: [v[s] for s in self.state] for k, v in self.snapshots.items()}
        rows = batch.out_rows if batch.out_rows is not None else [e - 1 for e in batch.cu_seqlens[1:]]
        return norm(x[rows], "final.norm")

    @torch.no_grad()
    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        cap = self.cfg.logit_softcap
        return cap * torch.tanh((hidden @ self.w["head"].t()).float() / cap)
