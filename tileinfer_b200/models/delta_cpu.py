"""PyTorch executor of Luvapel on a CPU: pages of keys and values, recurrent states and convolution tails in slots with
snapshots, variable-length batches, prefix reuse and swapping can be exercised by the engine without a GPU.  (The GPU executor
is `delta_b200.py`; nothing there falls back to this.)
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .luvapel import BRANCH_SCALE, DECAY_SCALE, LuvapelConfig, ParallelMixer
from .mixed_cpu import TorchMixedModel, turn_pairs
from .reference_cpu import Batch, rmsnorm
from .weights import fake_quant


class TorchDeltaModel(TorchMixedModel):
    """Cache pages, slots, snapshots, convolutions and windowed attention are those of the other mixed executor."""
    QUANTISED = (".q", ".k", ".v", ".g", ".o", ".r", ".a", ".b", ".w1", ".rg1", ".rg2", ".up", ".down")

    def __init__(self, cfg: LuvapelConfig, src, *, quant: str = "none", dtype=torch.float32, tp: int = 1, rank: int = 0, comm=None):
        super().__init__(cfg, src, quant="none", dtype=dtype, tp=tp, rank=rank, comm=comm)
        if quant == "w8a16":
            for n, w in self.w.items():
                if n.endswith(self.QUANTISED) and w.dim() == 2:
                    self.w[n] = fake_quant(w).to(dtype)

    def alloc_cache(self, num_blocks: int, block_size: int, num_slots: int):
        self.block_size = block_size
        n = num_blocks * block_size
        for i, L in enumerate(self.cfg.layers):
            m = L.mixer
            if not isinstance(m, ParallelMixer):
                self.state[i, "delta"] = torch.zeros(num_slots, m.heads, m.dim, m.dim)
                continue
            a, r = m.left, m.right
            self.pages[i] = tuple(torch.zeros(n, a.kv_heads, a.dim, dtype=self.dtype) for _ in range(2))
            self.state[i, "conv"] = torch.zeros(num_slots, r.taps - 1, 2 * r.kv_heads * r.dim + r.heads * r.vdim, dtype=self.dtype)
            self.state[i, "delta"] = torch.zeros(num_slots, r.heads, r.dim, r.vdim)

    # ---- mixers
    def _key_value_attention(self, i: int, a, p: str, h, batch: Batch):
        w, T, eps = self.w, h.shape[0], self.cfg.rms_eps
        head = lambda x, n: turn_pairs(rmsnorm(x.float(), w[f"{p}{n}.norm"], eps, one_plus=False), batch.positions, a.rot_dims, a.rot_base)
        k = (h @ w[p + "k"].t()).view(T, a.kv_heads, a.dim)
        self._store(self.pages[i][0], head(k, "k"), batch)
        self._store(self.pages[i][1], k, batch)
        q = head((h @ w[p + "q"].t()).view(T, a.heads, a.dim), "q") * w[p + "temp"].float()[:, None]
        o = self._attend(i, a, q, batch).reshape(T, -1) * torch.sigmoid((h @ w[p + "g"].t()).float())
        return o.to(self.dtype) @ w[p + "o"].t()

    def _recur(self, i: int, batch: Batch, T: int, step):
        """Runs `step(state, token) -> (state, output [heads, dv])` over every sequence from its slot's state."""
        key, out = (i, "delta"), None
        for s, t0, t1, first, points in self._sequences(batch):
            S = self.state[key][batch.state_slots[s]]
            for t in range(t0, t1):
                S, o = step(S, t)
                out = torch.empty(T, *o.shape) if out is None else out
                out[t] = o
                if first + t - t0 + 1 in points:
                    self._snapshot(s, first + t - t0 + 1, key, S)
            self.state[key][batch.state_slots[s]] = S
        return out

    def _unit(self, x):
        return x * torch.rsqrt((x * x).sum(-1, keepdim=True) + 1e-6)

    def _gated_delta(self, i: int, r, p: str, h, batch: Batch):
        w, T, dt = self.w, h.shape[0], self.dtype
        u = torch.cat([h @ w[p + n].t() for n in "qkv"], 1)
        u = F.silu(self._conv(i, u, torch.cat([w[f"{p}{n}.conv"] for n in "qkv"]), batch)).to(dt).float()
        q, k, v = u.split([r.kv_heads * r.dim, r.kv_heads * r.dim, r.heads * r.vdim], 1)
        spread = lambda x: self._unit(x.view(T, r.kv_heads, r.dim)).repeat_interleave(r.heads // r.kv_heads, 1)
        q, k, v = spread(q) * r.dim ** -0.5, spread(k), v.view(T, r.heads, r.vdim)
        beta = torch.sigmoid((h @ w[p + "b"].t()).float())
        g = torch.exp(-torch.exp(w[p + "A_log"].float()) * F.softplus((h @ w[p + "a"].t()).float() + w[p + "dt_bias"].float(), threshold=1e9))

        def step(S, t):
            S = S * g[t][:, None, None]
            new = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
            S = S + k[t][:, :, None] * new[:, None, :]
            return S, torch.einsum("hdv,hd->hv", S, q[t])
        o = self._recur(i, batch, T, step)
        o = rmsnorm(o, w[p + "norm"], self.cfg.rms_eps, one_plus=False).reshape(T, -1) * F.silu((h @ w[p + "g"].t()).float())
        return o.to(dt) @ w[p + "o"].t()

    def _general_delta(self, i: int, m, p: str, h, batch: Batch):
        w, T, heads = self.w, h.shape[0], lambda x: x.float().view(h.shape[0], m.heads, m.dim)
        r, k, v = (heads(h @ w[p + n].t()) for n in "rkv")
        z = torch.tanh((h @ w[p + "w1"].t()).float()) @ w[p + "w2"].float().t() + w[p + "w0"].float()
        decay = heads(torch.exp(-DECAY_SCALE * torch.sigmoid(z)))
        u = self._unit(k)
        gone = heads(torch.sigmoid((h @ w[p + "a"].t()).float() + w[p + "a.b"].float())) * u

        def step(S, t):
            read = torch.einsum("hdv,hd->hv", S, u[t])
            S = S * decay[t][:, :, None] - gone[t][:, :, None] * read[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
            return S, torch.einsum("hdv,hd->hv", S, r[t])
        o = self._recur(i, batch, T, step)
        one = torch.ones(m.dim)
        o = rmsnorm(o, one, self.cfg.rms_eps, one_plus=False).reshape(T, -1) * w[p + "norm"].float() * torch.sigmoid((h @ w[p + "g"].t()).float())
        return o.to(self.dtype) @ w[p + "o"].t()

    def _mixer(self, i: int, m, p: str, h, batch: Batch):
        if not isinstance(m, ParallelMixer):
            return self._general_delta(i, m, p, h, batch).float()
        left, right = self._key_value_attention(i, m.left, p + "left.", h, batch), self._gated_delta(i, m.right, p + "right.", h, batch)
        norm = lambda y, n: rmsnorm(y.float(), self.w[f"{p}{n}.out"], self.cfg.rms_eps, one_plus=False)
        return BRANCH_SCALE * (norm(left, "left") + norm(right, "right"))

    def _add(self, x, h, y, p: str, n: str):
        y = y * torch.sigmoid((h @ self.w[f"{p}rg{n}"].t()).float() + self.w[f"{p}rg{n}.b"].float())
        return x + rmsnorm(y, self.w[f"{p}norm{n}"], self.cfg.rms_eps, one_plus=False)

    @torch.no_grad()
    def forward(self, batch: Batch) -> torch.Tensor:
        """Normalised hidden states of the last token of every sequence (or of `batch.out_rows`)."""
        c, w = self.cfg, self.w
        x = w["embed"][batch.input_ids].float() * c.embedding_scale
        self.snapshots = {}
        for i, L in enumerate(c.layers):
            p = f"l{c.owner(i)}."
            h = x.to(self.dtype)
            x = self._add(x, h, self._mixer(i, L.mixer, p + "mix.", h, batch), p, "1")
            if L.mlp is not None:
                h = x.to(self.dtype)
                act = torch.relu(h @ w[p + "mlp.up"].t()) ** 2
                x = self._add(x, h, (act @ w[p + "mlp.down"].t()).float(), p, "2")
        self.snapshots = {k: [v[s] for s in self.state] for k, v in self.snapshots.items()}
        rows = batch.out_rows if batch.out_rows is not None else [e - 1 for e in batch.cu_seqlens[1:]]
        return rmsnorm(x[rows], w["final.norm"], c.rms_eps, one_plus=False).to(self.dtype)

    @torch.no_grad()
    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return (hidden @ self.w["head"].t()).float()
