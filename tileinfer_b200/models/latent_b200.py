"""Kabadra on one B200: weights in kernel layout, the paged cache of latents, the fused step.

A layer is parallel (mixer and feed-forward read the same norm and add to the same fp32 residual), so its products merge:
ONE input product gives [queries | latent | output gates | gate, up] and ONE output product over the concatenated
[heads | activated ff] columns adds both sublayers to the residual in its epilogue.  Per layer a decode step launches

  RMSNorm -> input product [clamped gated unit in the epilogue] -> latent norm + cache store -> W_uk absorbed into q
  -> attention over the paged latents [window, sink] -> W_uv and the output gate -> output product [fp32 residual add]

Sequences with many tokens in a step instead expand keys and values once per cached latent in reach (one tcgen05 product)
and run the windowed tcgen05 attention of `latent_prefill.cu`.  Head and latent sizes are padded to multiples of 64 with
zero weights, so any size runs.  quant: "bf16", "w8a16" (int8 input / output projections) or "fp32" (everything in 32
bits: plain FMA products, fp32 cache).
"""
from __future__ import annotations

import torch

from ..ops import functional as F
from ..ops.functional import LatentAttnParams, LinearW, ptr
from ..utils.trace import nvtx_end, nvtx_mark
from .kabadra import GLU_ALPHA, GLU_BIAS, KabadraConfig
from .products_b200 import Product, pad64, pad_to
from .runtime_b200 import DeviceRuntime, StepCtx

PAGE = 16


class _Layer:
    pass


class LatentLayers:
    """Launches of attention over paged latents, for executors with such layers.  A layer has heads, dp and vp (padded query
    and value heads), Rp (padded cache row), Ro (its leading columns that are values), window, scale, uk_t [H, Rp, dp],
    uv [H, vp, Ro], w_ukv (keys of all heads, then values; 16 bits) and, or None, sink and g_col (gate column)."""

    def _latent_rows(self, L):
        """The pages a layer attends to, [blocks, 16, Rp]."""
        raise NotImplementedError

    def _latent_nsplit(self, L, num_qg: int) -> int:
        return F.latent_nsplit(num_qg, L.heads, L.Rp, L.window) if not self.f32 and F.latent_attn_splits(L.Rp, L.Ro) else 1

    def _alloc_latent(self, x: StepCtx, T: int, num_qg: int, layers: list, new):
        x.short_rows = (0, T)               # rows [a, b) that hold every token of the split attention
        x.reach, x.latents = {}, {}         # window -> (cache slots in reach, query tiles) of the long portions
        if not (num_qg and layers):
            return
        x.q_abs = new(T * max(L.heads * L.Rp for L in layers), dtype=self.dtype, device=self.dev)
        x.o_lat = new(T * max(L.heads * L.Ro for L in layers), dtype=self.dtype, device=self.dev)
        part = max((F.latent_part_floats(num_qg, L.heads, L.Rp, ns) for L in layers if (ns := self._latent_nsplit(L, num_qg)) > 1), default=0)
        if part:
            x.lat_part = torch.empty(part, dtype=torch.float32, device=self.dev)
            x.lat_ml = torch.empty(part // 64 * 2, dtype=torch.float32, device=self.dev)

    def _attn_latent_short(self, L, x: StepCtx, proj, cat):
        """Decode tokens and short portions: absorbed queries against the paged latents."""
        a, b = x.short_rows
        T, H = x.T, L.heads
        q_abs, o_lat = x.q_abs[:T * H * L.Rp].view(T, H * L.Rp), x.o_lat[:T * H * L.Ro].view(T, H * L.Ro)
        F.head_product(proj[a:b], L.uk_t, q_abs[a:b])
        p = LatentAttnParams()
        p.q, p.cache, p.out, p.sink = ptr(q_abs), ptr(self._latent_rows(L)), ptr(o_lat), ptr(L.sink)
        p.block_tables, p.positions = ptr(x.block_tables), ptr(x.positions)
        p.qg_seq, p.qg_tok0, p.qg_ntok = ptr(x.qg[0]), ptr(x.qg[1]), ptr(x.qg[2])
        p.nsplit = self._latent_nsplit(L, x.num_qg)
        if p.nsplit > 1:
            p.o_part, p.ml_part = ptr(x.lat_part), ptr(x.lat_ml)
        p.H, p.R, p.Rp, p.Ro, p.max_blocks, p.num_qg = H, L.R, L.Rp, L.Ro, x.max_blocks, x.num_qg
        p.window, p.num_blocks, p.scale, p.status = L.window, self.num_blocks, L.scale, self.status
        F.latent_attn(p, self.f32)
        F.head_product(o_lat[a:b], L.uv, cat[a:b], gate=None if L.g_col is None else proj[a:b], gcol=L.g_col or 0)
        self._launches += 3 + (p.nsplit > 1)

    def _prepare_latent(self, x: StepCtx, batch, layers: list):
        """Which rows the split attention covers, and per window the cached rows in reach of the long portions of the step
        with their query tiles (see `latent_prefill`)."""
        bs, short, longs = self.block_size, [], []
        for s in range(batch.num_seqs):
            t0, t1 = batch.cu_seqlens[s], batch.cu_seqlens[s + 1]
            (longs if t1 - t0 >= self.PREFILL_ATTN_MIN_TOKENS else short).append((s, t0, t1))
        x.short_rows = (short[0][1], short[-1][2]) if short else (0, 0)
        for window in {L.window for L in layers} if longs else ():
            slots, tiles, base = [], [], 0
            for s, t0, t1 in longs:
                end = batch.context_lens[s]
                start = end - (t1 - t0)
                lo = max(0, start - window + 1)
                pos = torch.arange(lo, end)
                slots.append(torch.tensor(batch.block_tables[s], dtype=torch.long)[pos // bs] * bs + pos % bs)
                for a in range(t0, t1, 128):
                    p0, n = start + a - t0, min(128, t1 - a)
                    tiles.append((p0 + n - max(0, p0 - window + 1), a, n, p0, base, lo))
                base += end - lo
            tiles.sort(key=lambda t: -t[0])                    # most keys first
            x.reach[window] = (torch.cat(slots).to(self.dev, non_blocking=True),
                               torch.tensor([t[1:] for t in tiles], dtype=torch.int32).t().contiguous().to(self.dev, non_blocking=True))

    def _attn_latent_long(self, L, x: StepCtx, proj, cat):
        """Long portions of prompts: keys and values of every cached latent in reach, then windowed query tiles."""
        slots, tiles = x.reach[L.window]
        n, key = slots.numel(), (self._latent_rows(L).data_ptr(), L.window)
        if key not in x.latents:                               # layers that share latents share the gathered rows
            x.latents[key] = torch.empty(n, L.Rp, dtype=self.dtype, device=self.dev)
            F.latent_gather(self._latent_rows(L), slots, x.latents[key])
            self._launches += 1
        kv = torch.empty(n, L.w_ukv.N, dtype=self.dtype, device=self.dev)
        F.gemm_bf16(L.w_ukv, x.latents[key], out=kv)
        F.latent_prefill(proj, kv, tiles, cat, H=L.heads, dp=L.dp, vp=L.vp, window=L.window, scale=L.scale, sink=L.sink,
                         gate=None if L.g_col is None else proj, gcol=L.g_col or 0, status=self.status)
        self._launches += 2


class B200LatentModel(LatentLayers, DeviceRuntime):
    def __init__(self, cfg: KabadraConfig, src, *, quant="bf16", tp=1, rank=0, comm=None, config=None):
        assert torch.cuda.is_available(), "B200LatentModel needs a CUDA device"
        cfg.validate_tp(tp)
        F.L("base", "rows", "latent")              # load (or build) the kernel libraries now: fail loudly if they are missing
        self.cfg, self.tp, self.rank, self.comm, self.peer = cfg, tp, rank, comm, None
        self.dev = torch.device("cuda", torch.cuda.current_device())
        self.quant, self.f32 = quant, quant == "fp32"
        self.dtype = torch.float32 if self.f32 else torch.bfloat16
        self.W, self.Wp = cfg.hidden_size, pad64(cfg.hidden_size)
        self.vocab_start, self.v_local = 0, cfg.vocab_size
        self._build(src)
        torch.cuda.empty_cache()
        self.hkv = max(-(-L.heads // F.latent_rows(L.heads)) for L in self.layers)   # head groups per query token
        self.block_size, self.cache = PAGE, {}
        self.graphs, self.snapshots, self.host_steps = {}, {}, 0
        self.launches_per_decode_step = self._launches = 0
        # sequences with at least this many tokens in a step expand keys and values (tcgen05 tiles)
        tiled = not self.f32 and all(L.dp <= 256 and L.vp <= 256 for L in self.layers)
        self.PREFILL_ATTN_MIN_TOKENS = 32 if tiled else 1 << 30
        self.status = F.status_ptr()

    # ------------------------------------------------------------------ weights
    def _norm(self, w: torch.Tensor, n: int) -> torch.Tensor:
        return pad_to(w.float(), n).to(self.dev)

    def _build(self, src):
        c, dev, Wp = self.cfg, self.dev, self.Wp
        get = lambda name: src.get(name).to(dev)
        self.embed = pad_to(get("embed"), c.vocab_size, Wp).to(self.dtype).contiguous()
        self.pos = pad_to(get("pos"), c.max_position_embeddings, Wp).to(self.dtype).contiguous()
        self.embed_norm, self.final_norm = self._norm(get("embed.norm"), Wp), self._norm(get("final.norm"), Wp)
        self.layers = []
        for i, spec in enumerate(c.layers):
            m, p, L = spec.mixer, f"l{i}.", _Layer()
            L.heads, L.dim, L.vdim, L.R = m.heads, m.dim, m.vdim, m.kv_rank
            L.dp, L.vp, L.Rp = pad64(m.dim), pad64(m.vdim), pad64(m.kv_rank)
            L.window, L.scale = m.window, m.scale
            L.Ro, L.owner, L.stores = L.Rp, c.latent_layer(i), m.kv_from is None
            L.norm1 = self._norm(get(p + "norm1"), Wp)
            H = m.heads
            q = pad_to(get(p + "mix.q").view(H, m.dim, -1), H, L.dp, Wp).reshape(H * L.dp, Wp)
            rows = [q]
            if L.stores:
                L.kv_col = H * L.dp
                L.kv_norm = self._norm(get(p + "mix.dkv.norm"), L.Rp)
                rows.append(pad_to(get(p + "mix.dkv"), L.Rp, Wp))
            L.g_col = sum(r.shape[0] for r in rows)
            rows.append(pad_to(get(p + "mix.g"), -(-H // 8) * 8, Wp))
            L.n_proj = sum(r.shape[0] for r in rows)             # columns before the (gate, up) pairs
            o = pad_to(get(p + "mix.o").view(-1, H, m.vdim), Wp, H, L.vp).reshape(Wp, H * L.vp)
            L.n_mix, L.ff = H * L.vp, 0
            if spec.mlp is not None:
                L.ff, L.limit = pad64(spec.mlp.ff), spec.mlp.limit
                gate, up = pad_to(get(p + "mlp.gate"), L.ff, Wp), pad_to(get(p + "mlp.up"), L.ff, Wp)
                rows.append(torch.stack([gate, up], dim=1).reshape(2 * L.ff, Wp))
                o = torch.cat([o, pad_to(get(p + "mlp.down"), Wp, L.ff)], dim=1)
            L.w_in = Product(torch.cat(rows), self.quant, dev)
            L.w_out = Product(o, self.quant, dev)
            uk = pad_to(get(p + "mix.uk").view(H, m.dim, -1), H, L.dp, L.Rp)
            uv = pad_to(get(p + "mix.uv").view(H, m.vdim, -1), H, L.vp, L.Rp)
            L.uk_t = uk.transpose(1, 2).to(self.dtype).contiguous()          # [H, Rp, dp]
            L.uv = uv.to(self.dtype).contiguous()                            # [H, vp, Rp]
            if not self.f32:                                                 # rows [K of all heads | V of all heads]
                L.w_ukv = LinearW(torch.cat([uk.reshape(H * L.dp, L.Rp), uv.reshape(H * L.vp, L.Rp)]), False, dev)
            L.sink = get(p + "mix.sink").float().contiguous()
            self.layers.append(L)
        self.head = Product(pad_to(get("head"), c.vocab_size, Wp), "fp32" if self.f32 else "bf16", dev)

    def weight_bytes(self) -> int:
        """Bytes of weights a decode step streams."""
        n = self.head.nbytes()
        for L in self.layers:
            n += L.w_in.nbytes() + L.w_out.nbytes() + (L.uk_t.numel() + L.uv.numel()) * L.uv.element_size()
        return n

    # ------------------------------------------------------------------ cache: pages of 16 latents per owning layer
    def _bytes_per_block(self) -> int:
        return sum(PAGE * self.layers[i].Rp for i in self.cfg.latent_owners) * (4 if self.f32 else 2)

    cache_bytes_per_block = _bytes_per_block

    def auto_num_blocks(self, util, block_size, num_slots, max_num_seqs, max_model_len) -> int:
        free, total = torch.cuda.mem_get_info()
        n = int((free - (1.0 - util) * total - (2 << 30)) // self._bytes_per_block())
        n = min(n, max_num_seqs * (max_model_len // block_size + 2) + 64)
        if n < max_model_len // block_size + 2:
            raise RuntimeError(f"not enough GPU memory for one sequence of {max_model_len} tokens ({n} cache blocks)")
        return n

    def alloc_cache(self, num_blocks: int, block_size: int, num_slots: int):
        assert block_size == PAGE
        self.num_blocks = num_blocks
        self.cache = {i: torch.zeros(num_blocks, PAGE, self.layers[i].Rp, dtype=self.dtype, device=self.dev)
                      for i in self.cfg.latent_owners}

    def zero_state(self, slot: int):
        pass                                # a sequence has no state beside its cache blocks

    def state_out(self, slot: int):
        return None

    def state_in(self, slot: int, st):
        pass

    def blocks_out(self, block_ids: list):
        idx = torch.tensor(block_ids, dtype=torch.long, device=self.dev)
        dev = torch.cat([c[idx].flatten(1) for c in self.cache.values()], dim=1)
        host = self._pinned(dev.shape, dev.dtype)
        host.copy_(dev, non_blocking=True)
        return host

    def blocks_in(self, block_ids: list, data):
        idx = torch.tensor(block_ids, dtype=torch.long, device=self.dev)
        dev, at = data.to(self.dev, non_blocking=True), 0
        for c in self.cache.values():
            n = c[0].numel()
            c[idx] = dev[:, at:at + n].view(-1, *c.shape[1:])
            at += n
        if data.device.type == "cpu" and data.is_pinned():
            self._unpin(data)

    # ------------------------------------------------------------------ step
    def _alloc_ctx(self, T: int, S: int, max_blocks: int, num_qg: int, nsplit: int) -> StepCtx:
        x, dev, dt = self._alloc_inputs(T, S, max_blocks, num_qg, nsplit), self.dev, self.dtype
        # rows of padding sequences in a captured step are never written: zeros, so that they stay finite
        new = torch.zeros if T <= 256 else torch.empty
        x.x = new(T, self.Wp, dtype=torch.float32, device=dev)
        x.h = new(T, self.Wp, dtype=dt, device=dev)
        x.proj = new(T * max(L.n_proj for L in self.layers), dtype=dt, device=dev)
        x.cat = new(T * max(L.n_mix + L.ff for L in self.layers), dtype=dt, device=dev)
        self._alloc_latent(x, T, num_qg, self.layers, new)
        return x

    def _latent_rows(self, L):
        return self.cache[L.owner]

    def _prepare_step(self, x: StepCtx, batch):
        self._prepare_latent(x, batch, self.layers)

    def _run_layers(self, x: StepCtx):
        c, T = self.cfg, x.T
        F.embed_pos(x.ids, x.positions, self.embed, self.pos, self.embed_norm, x.x, self.W, c.rms_eps)
        self._launches += 1
        for i, L in enumerate(self.layers):
            nvtx_mark(f"layer {i}")
            proj = x.proj[:T * L.n_proj].view(T, L.n_proj)
            cat = x.cat[:T * (L.n_mix + L.ff)].view(T, L.n_mix + L.ff)
            F.rmsnorm_f32(x.x, L.norm1, x.h, self.W, c.rms_eps)
            if L.ff:
                ex = F.gemm_epilogue(out2=cat[:, L.n_mix:], n_split=L.n_proj, glu=(L.limit, GLU_ALPHA, GLU_BIAS))
                n = L.w_in(x.h, proj, F.GEPI_SPLIT_GLU, ex)
            else:
                n = L.w_in(x.h, proj, F.GEPI_STORE)
            if L.stores:
                F.latent_store(proj, L.kv_col, L.kv_norm, x.slot_mapping, self.cache[i], L.R, c.rms_eps)
                n += 1
            if x.num_qg:
                self._attn_latent_short(L, x, proj, cat)
            if x.reach:
                self._attn_latent_long(L, x, proj, cat)        # after the split attention, whose row range may span these
            n += L.w_out(cat, x.x, F.GEPI_RESID32, F.gemm_epilogue(resid32=x.x))
            self._launches += n + 1
        nvtx_end()
        return x.x

    def _lm_head(self, hidden, logits, n):
        h = torch.empty(n, self.Wp, dtype=self.dtype, device=self.dev)
        F.rmsnorm_f32(hidden, self.final_norm, h, self.W, self.cfg.rms_eps)
        self._launches += 1 + self.head(h, logits, F.GEPI_F32, F.gemm_epilogue(scale=self.cfg.logit_scale))

    def _status_ptr(self) -> int:
        return self.status

    def peer_status(self) -> int:
        return int(F._STATUS[0].item())
