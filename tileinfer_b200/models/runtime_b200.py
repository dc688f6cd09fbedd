"""What every model executor on the GPU shares: the variable-length eager step, CUDA-graph decode in batch-size
buckets, the vocabulary top-k and the sampling on the device.

A model adds its weights, its cache and `_alloc_ctx` / `_run_layers` / `_lm_head` (see `hybrid_b200.py` and
`latent_b200.py`); `_prepare_step` / `_finish_step` are for the work lists and by-products only it has.
Device half of the reference's ModelRunner (engine/model_runner.py:135-498).
"""
from __future__ import annotations

import gc

import torch

from ..ops import functional as F
from ..ops.functional import EditParams, SampleParams, TopkParams, ptr


class StepCtx:
    """Device tensors of one step (static for CUDA-graph buckets, fresh for eager steps)."""
    snap_rel = None
    snap_idx = None
    snap_state = None
    snap_conv = None
    num_snap = 0
    cu = None
    tiles = None            # [3, n] query tiles of the tcgen05 prefill attention (sequence, first token, tokens)
    ck = None               # [4, nc] chunk table of the chunked DeltaNet prefill (None: token-serial kernel)
    seq_ck = None


class DeviceRuntime:
    # ------------------------------------------------------------------ host copies of cache contents (swap)
    # pinned buffers, recycled by shape; the copies are asynchronous and ordered by the compute stream
    def _pinned(self, shape, dtype):
        pool = getattr(self, "_pin_pool", None)
        if pool is None:
            pool = self._pin_pool = {}
        free = pool.setdefault((tuple(shape), dtype), [])
        return free.pop() if free else torch.empty(tuple(shape), dtype=dtype, pin_memory=True)

    def _unpin(self, t):
        self._pin_pool.setdefault((tuple(t.shape), t.dtype), []).append(t)

    def take_snapshots(self):
        out, self.snapshots = self.snapshots, {}
        return out

    # ------------------------------------------------------------------ helpers
    def _topk_geometry(self, k: int):
        V = self.v_local
        max_chunks = min(128, 8192 // k)
        cs = -(-V // max_chunks)
        cs = max(256, -(-cs // 256) * 256)
        assert cs <= 4096, "vocabulary shard too large for the top-k kernel"
        return -(-V // cs), cs

    def _make_topk(self, logits, n, k, order=65000, per_cta=False):
        chunks, cs = self._topk_geometry(k)
        if per_cta:                      # candidates come from the arg-max epilogue of the GEMV: one per row and CTA
            chunks, cs = F.NUM_SMS, 0
        dev = self.dev
        t = StepCtx()
        t.ws_val = torch.empty(n * chunks * k, dtype=torch.float32, device=dev)
        t.ws_idx = torch.empty(n * chunks * k, dtype=torch.int32, device=dev)
        t.out_val = torch.empty(n, self.tp * k if self.peer is not None else k, dtype=torch.float32, device=dev)
        t.out_idx = torch.empty_like(t.out_val, dtype=torch.int32)
        p = TopkParams()
        p.logits, p.ws_val, p.ws_idx, p.out_val, p.out_idx = ptr(logits), ptr(t.ws_val), ptr(t.ws_idx), ptr(t.out_val), ptr(t.out_idx)
        p.M, p.V, p.ld, p.k, p.chunks, p.chunk_size = n, self.v_local, 0 if logits is None else logits.stride(0), k, chunks, cs
        p.vocab_start = self.vocab_start
        p.tp, p.rank, p.order, p.m_cap = 1, 0, order, 0
        if self.peer is not None:
            p.tp, p.rank, p.m_cap = self.tp, self.rank, self.peer.m_cap
            for r in range(self.tp):
                p.peer_buf[r] = self.peer.cand_ptrs[r]
            p.step_ptr, p.status, p.timeout_ns = self.peer.step_ptr, self.peer.status_ptr, self.peer.timeout_ns
        t.params = p
        return t

    def _lm_head(self, hidden, logits, n):
        """Final norm and vocabulary product of `n` residual rows -> fp32 logits (model-specific)."""
        raise NotImplementedError

    def _run_layers(self, x: StepCtx):
        """Every launch from the token embedding to the residual stream after the last layer (model-specific)."""
        raise NotImplementedError

    def _alloc_ctx(self, T: int, S: int, max_blocks: int, num_qg: int, nsplit: int) -> StepCtx:
        """Device tensors of a step (model-specific; see `_alloc_inputs`)."""
        raise NotImplementedError

    def _prepare_step(self, x: StepCtx, batch):
        """Model-specific work lists of an eager step."""

    def _finish_step(self, x: StepCtx):
        """Model-specific outputs of an eager step (state snapshots)."""

    def _tokens_per_group(self) -> int:
        """Query tokens per work item of the split-KV attention."""
        return 1

    def fused_argmax_ok(self, n: int, k: int) -> bool:
        """Whether the vocabulary product can keep the arg-max itself (no logits in memory)."""
        return False

    def _alloc_inputs(self, T: int, S: int, max_blocks: int, num_qg: int, nsplit: int) -> StepCtx:
        """The inputs every model's step has: tokens, positions, cache slots, block tables, query groups."""
        dev, x = self.dev, StepCtx()
        x.T, x.S, x.max_blocks, x.num_qg, x.nsplit = T, S, max_blocks, num_qg, nsplit
        x.ids = torch.zeros(T, dtype=torch.long, device=dev)
        x.positions = torch.zeros(T, dtype=torch.int32, device=dev)
        x.slot_mapping = torch.full((T,), -1, dtype=torch.long, device=dev)
        x.slots = torch.zeros(S, dtype=torch.int32, device=dev)
        x.block_tables = torch.zeros(S, max_blocks, dtype=torch.int32, device=dev)
        x.qg = torch.zeros(3, max(num_qg, 1), dtype=torch.int32, device=dev)      # seq, tok0, ntok
        return x

    def _topk_rows(self, logits, n, k):
        """Per-rank top-k (+ fused candidate exchange); rows in chunks of the peer buffer capacity."""
        cap = self.peer.m_cap if self.peer is not None else n
        outs = []
        for ci, m0 in enumerate(range(0, n, cap)):
            m = min(cap, n - m0)
            t = self._make_topk(logits[m0:m0 + m], m, k, order=65000 + ci)
            F.topk(t.params)
            self._launches += 2
            outs.append(t)
        return torch.cat([t.out_val for t in outs]), torch.cat([t.out_idx for t in outs])

    # ------------------------------------------------------------------ eager variable-length step
    PREFILL_ATTN_MIN_TOKENS = 16      # sequences with at least this many tokens in a step use the tcgen05 attention

    def _fill_ctx(self, x: StepCtx, batch, host=None):
        """Work lists of the two attention kernels: query groups of one or two tokens for the split-KV kernel
        (decode tokens, short chunks) and 128-token query tiles, longest context first, for the tcgen05 kernel."""
        S, T = batch.num_seqs, batch.cu_seqlens[-1]
        gt = self._tokens_per_group()
        qg_seq, qg_tok0, qg_ntok, tiles = [], [], [], []
        for s in range(S):
            t0, t1 = batch.cu_seqlens[s], batch.cu_seqlens[s + 1]
            if t1 - t0 >= self.PREFILL_ATTN_MIN_TOKENS:
                start = batch.context_lens[s] - (t1 - t0)
                for a in range(t0, t1, 128):
                    n = min(128, t1 - a)
                    tiles.append((start + (a - t0) + n, s, a, n))
                continue
            for a in range(t0, t1, gt):
                qg_seq.append(s); qg_tok0.append(a); qg_ntok.append(min(gt, t1 - a))
        tiles.sort(reverse=True)
        return qg_seq, qg_tok0, qg_ntok, tiles

    @torch.no_grad()
    def forward(self, batch):
        """Eager step over a flattened batch (prefill chunks and/or decode tokens).  Returns the
        residual-stream rows of the last token of every sequence (or of `batch.out_rows`); the final
        norm belongs to the vocabulary product."""
        dev = self.dev
        S, T = batch.num_seqs, batch.cu_seqlens[-1]
        qg_seq, qg_tok0, qg_ntok, tiles = self._fill_ctx(None, batch)
        nq = len(qg_seq)
        max_blocks = max(len(b) for b in batch.block_tables)
        nsplit = 1 if nq * self.hkv >= F.NUM_SMS else max(1, min(32, -(-8 * F.NUM_SMS // (max(nq, 1) * self.hkv))))
        x = self._alloc_ctx(T, S, max_blocks, nq, nsplit)
        x.ids.copy_(batch.input_ids, non_blocking=True)
        x.positions.copy_(batch.positions.to(torch.int32), non_blocking=True)
        x.slot_mapping.copy_(batch.slot_mapping, non_blocking=True)
        x.slots.copy_(torch.tensor(batch.state_slots, dtype=torch.int32), non_blocking=True)
        x.cu = torch.tensor(batch.cu_seqlens, dtype=torch.int32, device=dev)
        bt = torch.zeros(S, max_blocks, dtype=torch.int32)
        for s, b in enumerate(batch.block_tables):
            bt[s, :len(b)] = torch.tensor(b, dtype=torch.int32)
        x.block_tables.copy_(bt, non_blocking=True)
        if nq:
            x.qg.copy_(torch.tensor([qg_seq, qg_tok0, qg_ntok], dtype=torch.int32), non_blocking=True)
        if tiles:
            x.tiles = torch.tensor([[t[1] for t in tiles], [t[2] for t in tiles], [t[3] for t in tiles]],
                                   dtype=torch.int32).to(dev, non_blocking=True)
        self._prepare_step(x, batch)
        cur = self._run_layers(x)
        rows = batch.out_rows if batch.out_rows is not None else [c - 1 for c in batch.cu_seqlens[1:]]
        hidden = cur[torch.tensor(rows, dtype=torch.long, device=dev)]
        self._finish_step(x)
        self.host_steps += 1
        return hidden

    @torch.no_grad()
    def logits(self, hidden) -> torch.Tensor:
        n = hidden.shape[0]
        hidden = hidden.contiguous()
        out = torch.empty(n, self.v_local, dtype=torch.float32, device=self.dev)
        self._lm_head(hidden, out, n)
        return out

    # ------------------------------------------------------------------ CUDA-graph decode
    def capture_decode_graphs(self, max_num_seqs, max_graph_bs, max_model_len, padding_slot):
        self.padding_slot = padding_slot
        self.graph_max_blocks = max_model_len // 16 + 2
        top = min(max_num_seqs, max_graph_bs)
        if self.peer is not None:
            top = min(top, self.peer.m_cap)      # one candidate exchange per step covers m_cap rows
        self.buckets = []
        b = 1
        while b < top:
            self.buckets.append(b)
            b *= 2
        self.buckets.append(top)
        self.graph_pool = None
        for b in self.buckets:
            self._get_graph(b, 1, self.fused_argmax_ok(b, 1))

    def release_graphs(self):
        """Drop every captured decode graph (and the reference to the one replayed last).  Graphs that captured NCCL
        collectives (the non-fused tensor-parallel path) must be gone before the process group is destroyed: NCCL
        waits for them."""
        self.graphs.clear()
        self._last_graph = None
        gc.collect()

    def decode_graph(self, n: int, k: int = 1, edits: bool = False):
        """The captured decode step that serves `n` sequences with `k` candidates (captured on first use)."""
        B = next(b for b in self.buckets if b >= n)
        k = 1 if k <= 1 else 64
        return self._get_graph(B, k, not edits and self.fused_argmax_ok(B, k))

    def _get_graph(self, B: int, k: int, fa: bool = False):
        """fa: the lm_head product keeps only each CTA's arg-max (greedy rows without logit edits)."""
        key = (B, k, fa)
        g = self.graphs.get(key)
        if g is not None:
            return g
        dev = self.dev
        nsplit = max(1, min(32, -(-8 * F.NUM_SMS // (B * self.hkv))))
        base = next((v for kk, v in self.graphs.items() if kk[0] == B), None)
        g = StepCtx()
        if base is not None:      # same bucket, other k: share the input tensors
            g.x = base.x
            g.host = base.host
        else:
            g.x = self._alloc_ctx(B, B, self.graph_max_blocks, B, nsplit)
            x = g.x
            g.host = {
                "ids": torch.zeros(B, dtype=torch.long).pin_memory(),
                "positions": torch.zeros(B, dtype=torch.int32).pin_memory(),
                "slot_mapping": torch.full((B,), -1, dtype=torch.long).pin_memory(),
                "slots": torch.full((B,), self.padding_slot, dtype=torch.int32).pin_memory(),
                "block_tables": torch.zeros(B, self.graph_max_blocks, dtype=torch.int32).pin_memory(),
                "qg": torch.zeros(3, B, dtype=torch.int32).pin_memory(),
            }
            x.slots.fill_(self.padding_slot)
        x = g.x
        g.logits = None if fa else torch.zeros(B, self.v_local, dtype=torch.float32, device=dev)
        g.topk = self._make_topk(g.logits, B, k, per_cta=fa)
        g.k = k
        g.samp = self._make_sampler_state(g.logits if not fa else g.topk.out_val, B, g.topk)
        fused_sample = self.tp == 1 or self.peer is not None

        def body():
            cur = self._run_layers(x)
            if fa:
                self._lm_head_argmax(cur, g.topk, B)
            else:
                self._lm_head(cur, g.logits, B)
                F.logits_edit(g.samp.edit)             # rows without an edit slot leave at once
                F.topk(g.topk.params)
                self._launches += 3
            if fused_sample:
                F.sample(g.samp.sample)
                self._launches += 1

        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            body()                                   # warm-up (padding inputs touch only the padding slot)
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        if self.comm is not None:
            self.comm.barrier()
        self._launches = 0
        g.graph = torch.cuda.CUDAGraph()
        # objects of an earlier engine (old graphs, tensors) must not be finalised while the stream
        # captures: collect them now and keep the collector off until the capture ends
        gc.collect()
        gc_was_on = gc.isenabled()
        gc.disable()
        try:
            with torch.cuda.graph(g.graph, pool=self.graph_pool):
                body()
        finally:
            if gc_was_on:
                gc.enable()
        g.launches = self._launches
        self.launches_per_decode_step = g.launches
        if self.graph_pool is None:
            self.graph_pool = g.graph.pool()
        self.graphs[key] = g
        return g

    # ------------------------------------------------------------------ sampling on the device
    EDIT_SLOTS = 8          # rows of a step that may carry logit edits (penalty, bias, masks, grammar)
    PEN_CAP = 8192          # penalised token ids per row

    def _edit_buffers(self):
        """Device buffers of the logit-edit kernel, shared by all graphs and eager steps (stable addresses)."""
        e = getattr(self, "_edit", None)
        if e is None:
            dev, R = self.dev, self.EDIT_SLOTS
            e = self._edit = StepCtx()
            e.add_rows = torch.zeros(R, self.v_local, dtype=torch.float32, device=dev)
            e.meta = torch.zeros(3, R, dtype=torch.int32, device=dev)          # add_valid | pen_cnt | pen_rp (float bits)
            e.pen_ids = torch.zeros(R, self.PEN_CAP, dtype=torch.int32, device=dev)
            e.h_meta = torch.zeros(3, R, dtype=torch.int32).pin_memory()
            e.h_pen = torch.zeros(R, self.PEN_CAP, dtype=torch.int32).pin_memory()
            e.h_add = torch.zeros(R, self.v_local, dtype=torch.float32).pin_memory()
        return e

    def _make_sampler_state(self, logits, n, topk_state):
        """Parameter blocks of the edit and sample kernels for `n` rows whose candidates `topk_state` produces."""
        dev, e = self.dev, self._edit_buffers()
        t = StepCtx()
        t.fpar = torch.zeros(3, n, dtype=torch.float32, device=dev)            # temperature | top_p | u
        t.ipar = torch.full((2, n), -1, dtype=torch.int32, device=dev)         # top_k | edit slot
        t.h_fpar = torch.zeros(3, n, dtype=torch.float32).pin_memory()
        t.h_ipar = torch.full((2, n), -1, dtype=torch.int32).pin_memory()
        t.tok = torch.zeros(n + 1, dtype=torch.int32, device=dev)
        t.h_tok = torch.zeros(n + 1, dtype=torch.int32).pin_memory()
        ep = EditParams()
        ep.logits, ep.row_slot, ep.add_rows = ptr(logits), ptr(t.ipar[1]), ptr(e.add_rows)
        ep.add_valid, ep.pen_cnt, ep.pen_rp, ep.pen_ids = ptr(e.meta[0]), ptr(e.meta[1]), ptr(e.meta[2]), ptr(e.pen_ids)
        ep.M, ep.V, ep.ld, ep.pen_cap, ep.chunk = n, self.v_local, logits.stride(0), self.PEN_CAP, 8192
        t.edit = ep
        sp = SampleParams()
        sp.cand_val, sp.cand_idx = ptr(topk_state.out_val), ptr(topk_state.out_idx)
        sp.temperature, sp.top_p, sp.u, sp.top_k = ptr(t.fpar[0]), ptr(t.fpar[1]), ptr(t.fpar[2]), ptr(t.ipar[0])
        sp.out_tok, sp.status_src = ptr(t.tok), self._status_ptr()
        sp.M, sp.n_cand = n, topk_state.out_val.shape[1]
        t.sample = sp
        return t

    def _upload_sampling(self, t, n, spec):
        """Host -> device copies of a step's sampling parameters and logit edits (pinned staging, asynchronous)."""
        hf, hi = t.h_fpar, t.h_ipar
        hf[0].zero_()                                   # padding rows: greedy
        hi[1].fill_(-1)
        hf[0, :n] = torch.tensor(spec["temperature"], dtype=torch.float32)
        hf[1, :n] = torch.tensor(spec["top_p"], dtype=torch.float32)
        hf[2, :n] = torch.tensor(spec["u"], dtype=torch.float32)
        hi[0, :n] = torch.tensor(spec["top_k"], dtype=torch.int32)
        edits = spec.get("edits") or []
        if edits:
            e = self._edit_buffers()
            assert len(edits) <= self.EDIT_SLOTS
            for slot, (row, add, pen, rp) in enumerate(edits):
                hi[1, row] = slot
                e.h_meta[0, slot] = 0 if add is None else 1
                if add is not None:
                    e.h_add[slot].copy_(add)
                    e.add_rows[slot].copy_(e.h_add[slot], non_blocking=True)
                cnt = 0 if pen is None else min(len(pen), self.PEN_CAP)
                e.h_meta[1, slot] = cnt
                e.h_meta[2, slot] = torch.tensor([float(rp)], dtype=torch.float32).view(torch.int32)[0]
                if cnt:
                    e.h_pen[slot, :cnt] = pen[:cnt]
                    e.pen_ids[slot, :cnt].copy_(e.h_pen[slot, :cnt], non_blocking=True)
            e.meta.copy_(e.h_meta, non_blocking=True)
        t.fpar.copy_(hf, non_blocking=True)
        t.ipar.copy_(hi, non_blocking=True)

    def _read_tokens(self, t, n) -> list:
        """The step's only device -> host copy: n token ids and the communicator's status word."""
        t.h_tok.copy_(t.tok, non_blocking=True)
        torch.cuda.current_stream().synchronize()
        self.check_status(int(t.h_tok[t.tok.shape[0] - 1]))
        return t.h_tok[:n].tolist()

    def _decode_graph_step(self, batch, k: int, spec=None, keep_logits: bool = False):
        n = batch.num_seqs
        g = self.decode_graph(n, k, edits=keep_logits or bool(spec and spec.get("edits")))
        self._last_graph = g
        h, x = g.host, g.x
        h["ids"][:n] = batch.input_ids
        h["positions"][:n] = batch.positions
        h["slot_mapping"][:n] = batch.slot_mapping
        h["slot_mapping"][n:] = -1
        h["slots"][:n] = torch.tensor(batch.state_slots, dtype=torch.int32)
        h["slots"][n:] = self.padding_slot
        bt = h["block_tables"]
        for s, b in enumerate(batch.block_tables):
            bt[s, :len(b)] = torch.tensor(b, dtype=torch.int32)
        qg = h["qg"]
        qg[0, :n] = torch.arange(n, dtype=torch.int32)
        qg[1, :n] = torch.arange(n, dtype=torch.int32)
        qg[2, :n] = 1
        qg[2, n:] = 0
        x.ids.copy_(h["ids"], non_blocking=True)
        x.positions.copy_(h["positions"], non_blocking=True)
        x.slot_mapping.copy_(h["slot_mapping"], non_blocking=True)
        x.slots.copy_(h["slots"], non_blocking=True)
        x.block_tables.copy_(bt, non_blocking=True)
        x.qg.copy_(qg, non_blocking=True)
        if spec is not None:
            self._upload_sampling(g.samp, n, spec)
        if self.peer is not None:
            self.peer.tick()
        g.graph.replay()
        self.host_steps += 1
        return g.topk.out_val[:n], g.topk.out_idx[:n]

    def _graph_serves(self, batch) -> bool:
        """One token per sequence, and a captured bucket holds the step."""
        return bool(batch.cu_seqlens[-1] == batch.num_seqs and self.graphs and batch.num_seqs <= self.buckets[-1]
                    and max(len(b) for b in batch.block_tables) <= self.graph_max_blocks)

    @torch.no_grad()
    def step_logits(self, batch) -> torch.Tensor:
        """Runs the step the way generation does (captured graph for decode-only steps) and returns the fp32 logits
        of this rank's vocabulary shard at `batch.out_rows` (default: the last token of every sequence)."""
        rows = batch.out_rows if batch.out_rows is not None else [e - 1 for e in batch.cu_seqlens[1:]]
        if self._graph_serves(batch):
            self._decode_graph_step(batch, 1, keep_logits=True)
            return self._last_graph.logits[rows]
        hidden = self.forward(batch)
        return self.logits(hidden) if rows else torch.empty(0, self.v_local, device=self.dev)

    def _status_ptr(self) -> int:
        """Device word the kernels of this executor OR their error bits into."""
        return self.ctrl.data_ptr() + 4

    def check_status(self, status: int):
        """Raises when the device status word of a step is set: a bounded device wait ran out (a peer's flag or packet,
        an mbarrier) or a checked index was out of range, and whatever was computed after that is not to be trusted."""
        if status != 0:
            from ..parallel.watchdog import PeerLostError
            err = PeerLostError([])
            err.args = (f"device status word {status:#x}: a bounded wait ran out"
                        f"{' on a tensor-parallel peer' if self.peer is not None else ''} or an index check failed; "
                        "the tokens of this step are discarded",)
            raise err

    def _default_spec(self, n):
        return {"temperature": [0.0] * n, "top_k": [1] * n, "top_p": [1.0] * n, "u": [0.0] * n, "edits": []}

    @torch.no_grad()
    def forward_and_sample(self, batch, sample_rows, k: int, spec=None):
        """Runs the step and samples on the device.  Returns one token id per sampling row (a list of ints; the
        same on every tensor-parallel rank).  `spec`: per-row temperature / top_k / top_p / u lists and `edits`,
        a list of (row, additive logit row or None, sorted penalised local ids or None, penalty).  The step's only
        device -> host copy is the token ids plus the peer status word; a non-zero status raises PeerLostError."""
        assert k <= 64, "more than 64 candidates: use forward() + logits() + the host sampler"
        k = 1 if k <= 1 else 64
        n = len(sample_rows)
        if spec is None:
            spec = self._default_spec(n)
        fused = self.tp == 1 or self.peer is not None        # candidates of all ranks are on this device after top-k
        if n == batch.num_seqs and self._graph_serves(batch):
            vals, idx = self._decode_graph_step(batch, k, spec)
            if fused:
                return self._read_tokens(self._last_graph.samp, n)
        else:
            hidden = self.forward(batch)
            rows = torch.tensor(sample_rows, dtype=torch.long, device=self.dev)
            lg = self.logits(hidden[rows])
            if spec.get("edits"):
                t0 = StepCtx()
                t0.out_val = t0.out_idx = torch.empty(n, 1, device=self.dev)
                st = self._make_sampler_state(lg, n, t0)
                self._upload_sampling(st, n, spec)
                F.logits_edit(st.edit)
                self._launches += 1
            vals, idx = self._topk_rows(lg, n, k)
        if not fused:
            vals = torch.cat(self.comm.all_gather(vals.contiguous()), dim=-1)
            idx = torch.cat(self.comm.all_gather(idx.contiguous()), dim=-1)
        t1 = StepCtx()
        t1.out_val, t1.out_idx = vals.contiguous(), idx.contiguous()
        st = self._make_sampler_state(t1.out_val, n, t1)
        spec = dict(spec, edits=[])                    # edits were applied before the top-k
        self._upload_sampling(st, n, spec)
        F.sample(st.sample)
        self._launches += 1
        return self._read_tokens(st, n)

    def peer_status(self) -> int:
        return int(self.ctrl[1].item())
