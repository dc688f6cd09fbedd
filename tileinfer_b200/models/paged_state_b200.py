"""Cache pages and per-sequence state of the executors on the GPU whose layers have one, the other or both: `cache[key]` is a
tuple of page tensors [blocks, ...], `state[key]` a tensor [slots, ...].  Swapping, prefix snapshots and the work lists of
recurrent layers follow from these alone.
"""
from __future__ import annotations

import torch

from ..ops import functional as F
from .runtime_b200 import StepCtx

PAGE = 16


class PagedState:
    cache: dict
    state: dict

    # ------------------------------------------------------------------ pages and slots
    def _bytes_per_block(self) -> int:
        raise NotImplementedError

    def _state_bytes_per_slot(self) -> int:
        raise NotImplementedError

    def cache_bytes_per_block(self) -> int:
        return self._bytes_per_block()

    def auto_num_blocks(self, util, block_size, num_slots, max_num_seqs, max_model_len) -> int:
        free, total = torch.cuda.mem_get_info()
        budget = free - (1.0 - util) * total - num_slots * self._state_bytes_per_slot() - (6 << 30)        # room for the activations of a long step
        n = min(int(budget // max(1, self._bytes_per_block())), max_num_seqs * (max_model_len // block_size + 2) + 64)
        if n < max_model_len // block_size + 2:
            raise RuntimeError(f"not enough GPU memory for one sequence of {max_model_len} tokens ({n} cache blocks)")
        return n

    def zero_state(self, slot: int):
        for s in self.state.values():
            s[slot].zero_()

    def _to_host(self, parts):
        """One pinned host copy of the tensors, asynchronous and ordered by the stream (see `_pinned`)."""
        if not parts:
            return None
        dev = torch.cat(parts)
        host = self._pinned(dev.shape, dev.dtype)
        host.copy_(dev, non_blocking=True)
        return host

    def _done_with(self, data):
        if data.device.type == "cpu" and data.is_pinned():
            self._unpin(data)                          # later writers of the buffer are ordered after the copy from it

    def state_out(self, slot: int):
        return self._to_host([s[slot].flatten().float() for s in self.state.values()])

    def state_in(self, slot: int, st):
        """From a swapped-out state (pinned host memory) or a prefix snapshot (on the device, owned by the cache)."""
        if st is None:
            return
        dev, at = st.to(self.dev, non_blocking=True), 0
        for s in self.state.values():
            n = s[slot].numel()
            s[slot].copy_(dev[at:at + n].view(s[slot].shape))
            at += n
        self._done_with(st)

    def blocks_out(self, block_ids: list):
        idx = torch.tensor(block_ids, dtype=torch.long, device=self.dev)
        return self._to_host([t[idx].flatten() for pages in self.cache.values() for t in pages])

    def blocks_in(self, block_ids: list, data):
        if data is None:
            return
        idx, at = torch.tensor(block_ids, dtype=torch.long, device=self.dev), 0
        dev = data.to(self.dev, non_blocking=True)
        for t in (t for pages in self.cache.values() for t in pages):
            n = len(block_ids) * t[0].numel()
            t[idx] = dev[at:at + n].view(-1, *t.shape[1:])
            at += n
        self._done_with(data)

    # ------------------------------------------------------------------ recurrent layers in a step
    def _prepare_recurrence(self, x: StepCtx, batch, chunk_sizes, chunk_min_tokens: int):
        """State snapshots wanted in this step, and which sequences run the recurrence in chunks (of every size listed)."""
        S = batch.num_seqs
        points = batch.snapshot_at if batch.snapshot_at and any(batch.snapshot_at) else [[]] * S
        ns = max(len(p) for p in points)
        rel, idx = torch.zeros(S, max(ns, 1), dtype=torch.int32), torch.zeros(S, max(ns, 1), dtype=torch.int32)
        for s, pts in enumerate(points):
            start = batch.context_lens[s] - (batch.cu_seqlens[s + 1] - batch.cu_seqlens[s])
            for j, a in enumerate(pts):
                rel[s, j], idx[s, j] = a - start, len(x.snaps)
                x.snaps.append((s, a))
        if x.snaps:
            x.snap_rel, x.snap_idx, x.num_snap = rel.to(self.dev), idx.to(self.dev), ns
            x.snap_state = {k: torch.empty(len(x.snaps), *t.shape[1:], dtype=t.dtype, device=self.dev) for k, t in self.state.items()}
        lens = [b - a for a, b in zip(batch.cu_seqlens[:-1], batch.cu_seqlens[1:])]
        longs = [s for s in range(S) if lens[s] >= chunk_min_tokens] if chunk_sizes else []
        if longs:
            up = lambda v: torch.tensor(v, dtype=torch.int32).to(self.dev, non_blocking=True)
            x.short, x.longs = up([s for s in range(S) if lens[s] < chunk_min_tokens]), up(longs)
            entries = [{int(r): int(e) for r, e in zip(rel[s, :len(points[s])], idx[s])} for s in range(S)]
            for n in set(chunk_sizes):
                ck, rng = F.gla_chunk_table(batch.cu_seqlens, longs, n, entries)
                x.chunks[n] = (ck.to(self.dev, non_blocking=True), rng.to(self.dev, non_blocking=True))

    def _finish_step(self, x: StepCtx):
        for k, key in enumerate(x.snaps):                  # snapshots stay on the device
            self.snapshots[key] = torch.cat([t[k].flatten().float() for t in x.snap_state.values()])

    def peer_status(self) -> int:
        return int(F._STATUS[0].item())
