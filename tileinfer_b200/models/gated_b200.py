"""Gerivik on one B200: weights in kernel layout, paged keys and values, recurrent state slots, the fused step.

Per layer a decode step launches

  input product -> attention: rotation + unit heads + cache store -> paged attention with capped scores (+ merge)
                   gated linear attention: state step -> head norm + silu gate
  -> output product -> [norm, residual add, next norm, router product, routing, token rows to their experts]
  -> gate/up product [clamped gated unit in the epilogue] -> down product -> [weighted sum of the experts, norm, residual add, next layer's norm]

A layer that reuses another one's tensors shares its weights object and has a cache or state of its own.  Long portions of
prompts run the tcgen05 attention over the paged cache and the chunked form of the recurrence.  Head sizes are padded with
zero weights, so any size runs.  quant: "bf16", "w8a16" (int8 projections and experts) or "fp32" (everything in 32 bits).
The residual, norms, router scores, rotations, attention scores, decays and states are fp32 in every mode.
"""
from __future__ import annotations

import torch

from ..ops import functional as F
from ..ops.functional import AttnGeneralParams, AttnParams, GlaParams, RopeUnitParams, ptr
from ..utils.trace import nvtx_end, nvtx_mark
from .gerivik import GLU_ALPHA, GLU_BIAS, GerivikConfig
from .experts_b200 import ExpertLayers
from .paged_state_b200 import PAGE, PagedState
from .products_b200 import Product, pad64, pad_to
from .runtime_b200 import DeviceRuntime, StepCtx

LOG2E = 1.4426950408889634


def _pad_up(n: int, sizes) -> int:
    return next((s for s in sizes if s >= n), pad64(n))


def _heads(w: torch.Tensor, H: int, n: int, np_: int, Wp: int) -> torch.Tensor:
    """[H * n, W] rows of H heads -> [H * np_, Wp], each head padded with zero rows."""
    return pad_to(w.view(H, n, -1), H, np_, Wp).reshape(H * np_, Wp)


class _Weights:
    """Tensors of one layer in kernel layout (shared by the layers that reuse them)."""


class B200GatedModel(PagedState, ExpertLayers, DeviceRuntime):
    def __init__(self, cfg: GerivikConfig, src, *, quant="bf16", tp=1, rank=0, comm=None, config=None):
        assert torch.cuda.is_available(), "B200GatedModel needs a CUDA device"
        cfg.validate_tp(tp)
        F.L("base", "rows", "attention", "gla", "moe")     # load (or build) the kernel libraries now: fail loudly
        self.cfg, self.tp, self.rank, self.comm, self.peer = cfg, tp, rank, comm, None
        self.dev = torch.device("cuda", torch.cuda.current_device())
        self.quant, self.f32 = quant, quant == "fp32"
        self.dtype = torch.float32 if self.f32 else torch.bfloat16
        self.W, self.Wp = cfg.hidden_size, pad64(cfg.hidden_size)
        self.vocab_start, self.v_local = 0, cfg.vocab_size
        self._build(src)
        torch.cuda.empty_cache()
        attn = [self.layers[i] for i in cfg.attn_layers]
        self.hkv = max((L.G * L.rep for L in attn), default=1)            # blocks per query group of the split attention
        # heads wider than the tensor-core kernels take: every token of every layer is a query group of the split form
        tiled = not self.f32 and all(L.dp <= 256 and L.vp <= 256 for L in attn)
        self.PREFILL_ATTN_MIN_TOKENS = 16 if tiled else 1 << 30
        self._group_tokens = 2 if tiled and all(L.heads // (L.G * L.rep) * 2 <= 16 for L in attn) else 1
        # sequences with at least this many tokens in a step run the recurrence in chunks
        chunked = not self.f32 and all(F.gla_chunk_size(self.layers[i].dp) for i in cfg.gla_layers)
        self.gla_chunk_min_tokens = 32 if chunked else 1 << 30
        self.gla_ws = F.GlaWorkspace(self.dev)
        self.counters = F.moe_counters(max((L.mlp.experts for L in cfg.layers if L.mlp is not None), default=1), self.dev)
        self.block_size, self.cache, self.state = PAGE, {}, {}
        self.graphs, self.snapshots, self.host_steps = {}, {}, 0
        self.launches_per_decode_step = self._launches = 0
        self.status = F.status_ptr()

    def _tokens_per_group(self) -> int:
        return self._group_tokens

    # ------------------------------------------------------------------ weights
    def _norm(self, w: torch.Tensor, n: int) -> torch.Tensor:
        return pad_to(w.float(), n).to(self.dev)

    def _build(self, src):
        c, dev, Wp = self.cfg, self.dev, self.Wp
        get = lambda name: src.get(name).to(dev)
        self.embed = pad_to(get("embed"), c.vocab_size, Wp).to(self.dtype).contiguous()
        self.final_norm = self._norm(get("final.norm"), Wp)
        own = {i: self._build_layer(spec, f"l{i}.", get) for i, spec in enumerate(c.layers) if spec.weights_of is None}
        self.layers = [own[c.owner(i)] for i in range(c.num_layers)]
        self.owned = list(own.values())
        self.head = Product(pad_to(get("head"), c.vocab_size, Wp), "fp32" if self.f32 else "bf16", dev)

    def _build_layer(self, spec, p: str, get) -> _Weights:
        dev, Wp, L, m = self.dev, self.Wp, _Weights(), spec.mixer
        L.norm1, L.norm1b = self._norm(get(p + "norm1"), Wp), self._norm(get(p + "norm1b"), Wp)
        L.heads, L.is_gla, q = m.heads, spec.is_gla, p + "mix."
        if spec.is_gla:
            L.G, L.dp, L.vp = m.heads, _pad_up(m.dim, F.GLA_KEY_SIZES), pad64(m.vdim)
            if L.dp not in F.GLA_KEY_SIZES:
                raise ValueError(f"gated linear attention takes keys of at most {F.GLA_KEY_SIZES[-1]} per head, got {m.dim}")
        else:
            sizes = (64, 128, 256) if not self.f32 and max(m.dim, m.vdim) <= 256 else ()
            L.G, L.dp, L.vp = m.kv_heads, _pad_up(m.dim, sizes), _pad_up(m.vdim, sizes)
            if max(L.dp, L.vp) > 1024:
                raise ValueError(f"attention takes heads of at most 1024, got {max(m.dim, m.vdim)}")
            G = m.heads // m.kv_heads                        # query heads of a block: at most 16
            L.rep = G // max(d for d in range(1, 17) if G % d == 0)
            inv = [m.rot_base ** (-2.0 * i / m.rot_dims) for i in range(m.rot_dims // 2)]
            L.inv_freq = torch.tensor(inv or [0.0], dtype=torch.float64).float().to(dev)
        H, G = m.heads, L.G
        rows = [_heads(get(q + "q"), H, m.dim, L.dp, Wp), _heads(get(q + "k"), G, m.dim, L.dp, Wp), _heads(get(q + "v"), G, m.vdim, L.vp, Wp)]
        L.k_col, L.v_col = H * L.dp, (H + G) * L.dp
        if spec.is_gla:
            L.R, L.g_col = m.decay_rank, L.v_col + H * L.vp
            L.a_col = L.g_col + H * L.vp
            rows += [_heads(get(q + "g"), H, m.vdim, L.vp, Wp), pad_to(get(q + "a1"), -(-L.R // 8) * 8, Wp)]
            L.a2 = pad_to(get(q + "a2").view(H, m.dim, L.R), H, L.dp, L.R).reshape(H * L.dp, L.R).t().float().contiguous()
            L.a2_bias = pad_to(get(q + "a2.b").view(H, m.dim), H, L.dp).flatten().float().contiguous()
            L.head_norm = self._norm(get(q + "norm"), L.vp)
        L.w_in = Product(torch.cat(rows), self.quant, dev)
        L.n_proj, L.n_mix = L.w_in.N, H * L.vp
        L.w_o = Product(pad_to(get(q + "o").view(-1, H, m.vdim), Wp, H, L.vp).reshape(Wp, L.n_mix), self.quant, dev)
        L.moe = None
        if spec.mlp is not None:
            L.norm2, L.norm2b = self._norm(get(p + "norm2"), Wp), self._norm(get(p + "norm2b"), Wp)
            self._build_experts(L, spec.mlp, p + "mlp.", get, (spec.mlp.limit, GLU_ALPHA, GLU_BIAS), get(p + "mlp.correction").float().contiguous())
        return L

    def weight_bytes(self, tokens: int = 1) -> int:
        """Bytes of weights a decode step of `tokens` tokens streams (experts: at most top per token and layer)."""
        n = self.head.nbytes()
        for L in self.layers:
            n += L.w_in.nbytes() + L.w_o.nbytes()
            if L.moe is not None:
                n += self._expert_bytes(L, tokens)
        return n

    # ------------------------------------------------------------------ cache pages and state slots
    def _bytes_per_block(self) -> int:
        return sum(PAGE * L.G * (L.dp + L.vp) for L in (self.layers[i] for i in self.cfg.attn_layers)) * (4 if self.f32 else 2)

    def _state_bytes_per_slot(self) -> int:
        return sum(L.heads * L.dp * L.vp * 4 for L in (self.layers[i] for i in self.cfg.gla_layers))

    def alloc_cache(self, num_blocks: int, block_size: int, num_slots: int):
        assert block_size == PAGE
        self.num_blocks = num_blocks
        new = lambda dt, *s: torch.zeros(*s, dtype=dt, device=self.dev)
        for i in self.cfg.attn_layers:
            L = self.layers[i]
            self.cache[i] = (new(self.dtype, num_blocks, L.G, PAGE, L.dp), new(self.dtype, num_blocks, L.G, L.vp, PAGE))
        for i in self.cfg.gla_layers:
            L = self.layers[i]
            self.state[i] = new(torch.float32, num_slots, L.heads, L.dp, L.vp)

    # ------------------------------------------------------------------ step
    def _alloc_ctx(self, T: int, S: int, max_blocks: int, num_qg: int, nsplit: int) -> StepCtx:
        x, dev, dt, Ls = self._alloc_inputs(T, S, max_blocks, num_qg, nsplit), self.dev, self.dtype, self.owned
        # rows of padding sequences in a captured step are never written by the mixers: zeros, so that they stay finite
        new = torch.zeros if T <= 256 else torch.empty
        x.x = new(T, self.Wp, dtype=torch.float32, device=dev)
        x.h, x.y = new(T, self.Wp, dtype=dt, device=dev), new(T, self.Wp, dtype=dt, device=dev)
        x.proj = new(T * max(L.n_proj for L in Ls), dtype=dt, device=dev)
        x.mix = new(T * max(L.n_mix for L in Ls), dtype=dt, device=dev)
        attn, gla = [L for L in Ls if not L.is_gla], [L for L in Ls if L.is_gla]
        if attn:
            x.q = new(T * max(L.heads * L.dp for L in attn), dtype=dt, device=dev)
            if num_qg and not self.f32:
                items = max(num_qg * L.G * L.rep * nsplit * (L.vp if L.vp <= 256 else 0) for L in attn)
                x.o_part = torch.empty(items * 16, dtype=torch.float32, device=dev)
                x.ml_part = torch.empty(items // 64 * 32, dtype=torch.float32, device=dev)
        if gla:
            x.o = new(T * max(L.n_mix for L in gla), dtype=torch.float32, device=dev)
        self._alloc_experts(x, T, [L for L in Ls if L.moe is not None], new)
        x.snaps, x.chunks, x.short = [], {}, None          # chunks: chunk size -> (table, ranges); short: the other sequences
        return x

    def _prepare_step(self, x: StepCtx, batch):
        if self.cfg.gla_layers:
            self._prepare_recurrence(x, batch, [F.gla_chunk_size(self.layers[i].dp) for i in self.cfg.gla_layers], self.gla_chunk_min_tokens)

    def _rotate_and_store(self, i: int, L, x: StepCtx, proj):
        """Rotated unit heads of the queries (returned) and of the keys, and the values, into the cache pages."""
        m, (kc, vc), T = self.cfg.layers[i].mixer, self.cache[i], x.T
        q = x.q[:T * L.heads * L.dp].view(T, L.heads * L.dp)
        r = RopeUnitParams()
        r.proj, r.inv_freq, r.positions, r.slot_mapping = ptr(proj), ptr(L.inv_freq), ptr(x.positions), ptr(x.slot_mapping)
        r.q_out, r.kcache, r.vcache, r.status = ptr(q), ptr(kc), ptr(vc), self.status
        r.T, r.ld, r.q_col, r.k_col, r.v_col, r.H, r.G = T, proj.stride(0), 0, L.k_col, L.v_col, L.heads, L.G
        r.dim, r.dp, r.vp, r.half, r.num_blocks, r.eps = m.dim, L.dp, L.vp, m.rot_dims // 2, self.num_blocks, self.cfg.rms_eps
        F.rope_unit(r, self.f32)
        self._launches += 1
        return q

    def _attention(self, i: int, L, x: StepCtx, proj, mix):
        m, (kc, vc) = self.cfg.layers[i].mixer, self.cache[i]
        q = self._rotate_and_store(i, L, x, proj)
        if x.num_qg and (self.f32 or max(L.dp, L.vp) > 256):
            a = AttnGeneralParams()
            a.q, a.kcache, a.vcache, a.block_tables, a.positions = ptr(q), ptr(kc), ptr(vc), ptr(x.block_tables), ptr(x.positions)
            a.qg_seq, a.qg_tok0, a.qg_ntok, a.out, a.status = ptr(x.qg[0]), ptr(x.qg[1]), ptr(x.qg[2]), ptr(mix), self.status
            a.H, a.G, a.dp, a.vp, a.max_blocks, a.num_qg, a.num_blocks = L.heads, L.G, L.dp, L.vp, x.max_blocks, x.num_qg, self.num_blocks
            a.ldo, a.scale, a.softcap = mix.stride(0), m.scale, m.softcap
            F.attn_general(a, self.f32)
            self._launches += 1
        elif x.num_qg:
            a = AttnParams()
            a.q, a.kcache, a.vcache, a.block_tables, a.positions = ptr(q), ptr(kc), ptr(vc), ptr(x.block_tables), ptr(x.positions)
            a.qg_seq, a.qg_tok0, a.qg_ntok = ptr(x.qg[0]), ptr(x.qg[1]), ptr(x.qg[2])
            a.o_part, a.ml_part, a.out, a.status = ptr(x.o_part), ptr(x.ml_part), ptr(mix), self.status
            a.hq, a.hkv, a.rep, a.max_blocks, a.nsplit, a.num_qg, a.num_blocks = L.heads, L.G, L.rep, x.max_blocks, x.nsplit, x.num_qg, self.num_blocks
            a.cap_in, a.cap_out = 2.0 * m.scale / m.softcap * LOG2E, m.softcap * LOG2E
            F.attn_paged(a, L.dp, L.vp)
            self._launches += 2
        if x.tiles is not None:
            # unit heads bound q.k (Cauchy-Schwarz; with room for the rounding of both to bf16)
            F.attn_prefill(q, kc, vc, self.num_blocks, x.block_tables, x.positions, x.tiles, None, mix, hq=L.heads, hkv=L.G, D=L.dp,
                           DV=L.vp, max_blocks=x.max_blocks, ld=0, scale=m.scale, softcap=m.softcap, qk_max=1.02 * m.dim)
            self._launches += 1

    def _gla_params(self, i: int, L, x: StepCtx, proj, mix) -> GlaParams:
        m, p = self.cfg.layers[i].mixer, GlaParams()
        p.proj, p.a2, p.a2_bias, p.norm, p.state = ptr(proj), ptr(L.a2), ptr(L.a2_bias), ptr(L.head_norm), ptr(self.state[i])
        p.slots, p.cu, p.o, p.out = ptr(x.slots), ptr(x.cu), ptr(x.o), ptr(mix)
        if x.snaps:
            p.snap_rel, p.snap_idx, p.snap, p.num_snap = ptr(x.snap_rel), ptr(x.snap_idx), ptr(x.snap_state[i]), x.num_snap
        p.ld, p.ldo, p.H, p.R, p.vdim = proj.stride(0), mix.stride(0), L.heads, L.R, m.vdim
        p.q_col, p.k_col, p.v_col, p.g_col, p.a_col = 0, L.k_col, L.v_col, L.g_col, L.a_col
        p.q_scale, p.inv_tau, p.eps = m.dim ** -0.5, 1.0 / m.tau, self.cfg.rms_eps
        return p

    def _gla(self, i: int, L, x: StepCtx, proj, mix):
        p = self._gla_params(i, L, x, proj, mix)
        if x.short is not None:
            ck, rng = x.chunks[F.gla_chunk_size(L.dp)]
            p.ck_seq, p.ck_tok0, p.ck_ntok, p.ck_snap = (ptr(r) for r in ck)
            p.long_seq, p.long_ck, p.nc, p.num_long = ptr(x.longs), ptr(rng), ck.shape[1], x.longs.numel()
            p.g_ws, p.s_ws = (ptr(w) for w in self.gla_ws.get(p.nc, L.heads, L.dp, L.vp))
            F.gla_chunked(p, L.dp, L.vp)
            p.seqs = ptr(x.short)
            self._launches += 3
        num = x.S if x.short is None else x.short.numel()
        if num:
            F.gla_step(p, num, L.dp, L.vp, self.f32)
        F.gla_finish(p, x.T, L.vp, self.f32)
        self._launches += 1 + bool(num)

    def _run_layers(self, x: StepCtx):
        c, T = self.cfg, x.T
        F.embed_pos(x.ids, x.positions, self.embed, None, None, x.x, self.W, c.rms_eps, scale=c.embedding_scale)
        F.rmsnorm_f32(x.x, self.layers[0].norm1, x.h, self.W, c.rms_eps)
        self._launches += 2
        for i, L in enumerate(self.layers):
            nvtx_mark(f"layer {i}")
            proj, mix = x.proj[:T * L.n_proj].view(T, L.n_proj), x.mix[:T * L.n_mix].view(T, L.n_mix)
            n = L.w_in(x.h, proj, F.GEPI_STORE)
            (self._gla if L.is_gla else self._attention)(i, L, x, proj, mix)
            n += L.w_o(mix, x.y, F.GEPI_STORE)
            after = self.layers[i + 1].norm1 if i + 1 < len(self.layers) else None
            self._launches += n
            if L.moe is None:
                F.resid_norm(x.y, x.x, L.norm1b, x.h, after, self.W, c.rms_eps)
                self._launches += 1
            else:
                g, rows = self._norm_and_route(L, x, x.y, L.norm1b)
                self._experts(L, x, g, rows)
                F.resid_norm(rows, x.x, L.norm2b, x.h, after, self.W, c.rms_eps, routed=g)
                self._launches += 1
        nvtx_end()
        return x.x

    def _lm_head(self, hidden, logits, n):
        h = torch.empty(n, self.Wp, dtype=self.dtype, device=self.dev)
        F.rmsnorm_f32(hidden, self.final_norm, h, self.W, self.cfg.rms_eps)
        self._launches += 1 + self.head(h, logits, F.GEPI_F32)

    def _status_ptr(self) -> int:
        return self.status
