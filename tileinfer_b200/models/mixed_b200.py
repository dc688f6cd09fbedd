"""Nogidra on one B200: weights in kernel layout, pages of keys, values and latents, slots of recurrent states and convolution
tails, the fused step.

Per layer a decode step launches

  input product -> attention:  convolutions + query temperature + cache store -> paged attention [window, slopes] (+ merge, gate)
                   latent:     rotation + latent norm + cache store -> W_uk -> attention over latents (+ merge) -> W_uv
                   parallel:   norms + rotation + cache store -> paged attention (+ merge), and
                               convolution + silu -> state step -> gate + group norm
  -> output product [fp32 residual add] -> norm, or [norm, router product, routing, token rows to their experts]
  -> gate/up product [gated unit in the epilogue] -> down product [residual add; experts: their weighted sum with the next norm]

The two halves of a parallel mixer are one input product and one output product; their factors go into the attention's merge
and the group norm's weights.  The rotated key part of a latent layer is stored behind the latent, and W_uk is extended by
an identity block, so that one row is key (all of it) and value (the latent).  Long portions of prompts run the tcgen05
attention kernels and the chunked form of the recurrence.  Head, latent and state sizes are padded with zero weights, so any
size runs.  quant: "bf16", "w8a16" (int8 projections and experts) or "fp32" (everything in 32 bits).  The residual, norms,
router, angles, attention scores, step sizes, decays and states are fp32 in every mode.
"""
from __future__ import annotations

import math

import torch

from ..ops import functional as F
from ..ops.functional import LinearW, NormRopeParams, SsdParams, ptr
from ..utils.trace import nvtx_end, nvtx_mark
from .attention_b200 import AttentionLayers, head_rows, pad8, pad_up
from .conv_b200 import ConvLayers
from .experts_b200 import ExpertLayers
from .latent_b200 import LatentLayers
from .nogidra import ConvAttention, DenseGlu, NogidraConfig, ParallelMixer, RotaryLatent
from .paged_state_b200 import PAGE, PagedState
from .products_b200 import Product, pad64, pad_to
from .runtime_b200 import DeviceRuntime, StepCtx

SILU_UNIT = (math.inf, 1.0, 0.0)        # g sigmoid(g) u: limit, alpha, bias


class _Layer:
    attn = ssm = False                   # keys and values in pages; a recurrent state
    latent = None
    moe, ff = None, 0


class B200MixedModel(PagedState, AttentionLayers, ConvLayers, ExpertLayers, LatentLayers, DeviceRuntime):
    def __init__(self, cfg: NogidraConfig, src, *, quant="bf16", tp=1, rank=0, comm=None, config=None):
        assert torch.cuda.is_available(), "B200MixedModel needs a CUDA device"
        cfg.validate_tp(tp)
        kinds = {type(L.mixer) for L in cfg.layers}
        moe = any(L.mlp is not None and not isinstance(L.mlp, DenseGlu) for L in cfg.layers)
        # load (or build) the kernel libraries the layers need now: fail loudly
        F.L("base", "rows", *(["latent"] if RotaryLatent in kinds else []), *(["attention", "conv"] if kinds - {RotaryLatent} else []),
            *(["ssd"] if ParallelMixer in kinds else []), *(["moe"] if moe else []))
        self.cfg, self.tp, self.rank, self.comm, self.peer = cfg, tp, rank, comm, None
        self.dev = torch.device("cuda", torch.cuda.current_device())
        self.quant, self.f32 = quant, quant == "fp32"
        self.dtype = torch.float32 if self.f32 else torch.bfloat16
        self.W, self.Wp = cfg.hidden_size, pad64(cfg.hidden_size)
        self.vocab_start, self.v_local = 0, cfg.vocab_size
        self._build(src)
        torch.cuda.empty_cache()
        self.attn_layers = [L for L in self.layers if L.attn]
        self.latent_layers = [L for L in self.layers if L.latent]
        self.ssm_layers = [L for L in self.layers if L.ssm]
        self.hkv = max((L.G * L.rep for L in self.attn_layers), default=1)            # blocks per query group of the split attention
        # heads wider than the tensor-core kernels take: every token of every layer is a query of the split forms
        tiled = not self.f32 and all(L.dp <= 256 and L.vp <= 256 for L in self.layers)
        self.PREFILL_ATTN_MIN_TOKENS = 32 if tiled else 1 << 30
        # sequences with at least this many tokens in a step run the recurrence in chunks
        chunked = not self.f32 and all(F.ssd_chunk_size(L.Np) for L in self.ssm_layers)
        self.ssd_chunk_min_tokens = 32 if chunked else 1 << 30
        self.ssd_ws = F.SsdWorkspace(self.dev)
        self.counters = F.moe_counters(max((L.moe.experts for L in self.layers if L.moe is not None), default=1), self.dev)
        self.block_size, self.cache, self.state = PAGE, {}, {}
        self.graphs, self.snapshots, self.host_steps = {}, {}, 0
        self.launches_per_decode_step = self._launches = 0
        self.status = F.status_ptr()

    # ------------------------------------------------------------------ weights
    def _vec(self, w: torch.Tensor, n: int) -> torch.Tensor:
        return pad_to(w.float(), n).to(self.dev)

    def _build(self, src):
        c, dev, Wp = self.cfg, self.dev, self.Wp
        get = lambda name: src.get(name).to(dev)
        self.embed = pad_to(get("embed"), c.vocab_size, Wp).to(self.dtype).contiguous()
        self.final_norm = self._vec(1.0 + get("final.norm").float(), Wp)
        self.layers = [self._build_layer(i, spec, f"l{i}.", get) for i, spec in enumerate(c.layers)]
        self.head = Product(pad_to(get("head"), c.vocab_size, Wp), "fp32" if self.f32 else "bf16", dev)

    def _build_layer(self, i: int, spec, p: str, get) -> _Layer:
        L, Wp = _Layer(), self.Wp
        L.index, L.spec = i, spec.mixer
        L.norm1 = self._vec(1.0 + get(p + "norm1").float(), Wp)
        build = {ConvAttention: self._build_conv_attention, RotaryLatent: self._build_latent, ParallelMixer: self._build_parallel}
        rows, out, bias = build[type(spec.mixer)](L, spec.mixer, p + "mix.", get)
        L.w_in = Product(pad_to(rows, rows.shape[0], Wp), self.quant, self.dev)
        L.w_o = Product(pad_to(out, Wp, out.shape[1]), self.quant, self.dev)
        L.n_proj, L.n_mix, L.in_bias = L.w_in.N, out.shape[1], None if bias is None else self._vec(bias, L.w_in.N)
        if spec.mlp is None:
            return L
        L.norm2 = self._vec(1.0 + get(p + "norm2").float(), Wp)
        if isinstance(spec.mlp, DenseGlu):
            self._build_dense(L, spec.mlp, p + "mlp.", get)
        else:
            self._build_experts(L, spec.mlp, p + "mlp.", get, SILU_UNIT)
        return L

    def _build_dense(self, L, f: DenseGlu, p: str, get):
        L.ff = pad64(f.ff)
        pair = lambda a, b: torch.stack([a, b], dim=1).flatten(0, 1)
        g, u = (pad_to(get(p + n), L.ff, self.Wp) for n in ("gate", "up"))
        L.w_up, L.up_bias = Product(pair(g, u), self.quant, self.dev), pair(self._vec(get(p + "gate.b"), L.ff), self._vec(get(p + "up.b"), L.ff)).contiguous()
        L.w_down, L.down_bias = Product(pad_to(get(p + "down"), self.Wp, L.ff), self.quant, self.dev), self._vec(get(p + "down.b"), self.Wp)

    def _qkv(self, L, m, get, suffix=""):
        """The tensors q, k and v with their heads padded, one below the other."""
        return torch.cat([head_rows(get(f"q{suffix}"), m.heads, m.dim, L.dp), head_rows(get(f"k{suffix}"), m.kv_heads, m.dim, L.dp),
                          head_rows(get(f"v{suffix}"), m.kv_heads, m.vdim, L.vp)])

    def _build_conv_attention(self, L, m: ConvAttention, p: str, get):
        self._attention_sizes(L, m)
        q = lambda n: get(p + n)
        L.conv_col, L.taps, L.C = 0, m.taps, L.v_col + L.G * L.vp
        L.conv_w, L.conv_b = self._qkv(L, m, q, ".conv").t().float().contiguous(), None
        L.g_col, L.slopes = L.C, torch.tensor(m.slopes(), dtype=torch.float32, device=self.dev)
        gate = q("g")
        rows = torch.cat([self._qkv(L, m, q), pad_to(gate, pad8(m.heads), gate.shape[1])])
        return rows, self._out_columns(q("o"), m.heads, m.vdim, L.vp), None

    def _build_latent(self, L, m: RotaryLatent, p: str, get):
        H, R, P, dev = m.heads, m.kv_rank, m.rot_dim, self.dev
        L.latent, L.heads, L.dim, L.R = True, H, m.dim, R
        L.dp, L.vp, L.Rp, L.Ro = pad64(m.dim + P), pad64(m.vdim), pad64(R + P), pad64(R)
        if L.Rp > 2048:
            raise ValueError(f"a latent with its rotated part may have 2048 columns, got {R + P}")
        L.window, L.scale, L.sink, L.g_col = m.window, m.scale, None, None
        L.inv_freq, L.kv_norm = self._angles(m.rot_base, P), self._vec(get(p + "dkv.norm"), R)
        q, dkv = get(p + "q"), get(p + "dkv")
        L.kv_col = H * L.dp
        rows = torch.cat([head_rows(q, H, m.dim + P, L.dp), pad_to(dkv, pad64(R + P), dkv.shape[1])])
        # a query head [plain | turned] meets a cache row [latent | turned key part]: W_uk for the first, an identity for the second
        uk = pad_to(get(p + "uk").float().view(H, m.dim, R), H, L.dp, L.Rp)
        uk[:, m.dim:m.dim + P, R:R + P] = torch.eye(P, device=dev)
        uv = pad_to(get(p + "uv").float().view(H, m.vdim, R), H, L.vp, L.Rp)
        L.uk_t = uk.transpose(1, 2).to(self.dtype).contiguous()                  # [H, Rp, dp]
        L.uv = uv[..., :L.Ro].to(self.dtype).contiguous()                        # [H, vp, Ro]
        if not self.f32:                                                         # rows [K of all heads | V of all heads]
            L.w_ukv = LinearW(torch.cat([uk.reshape(H * L.dp, L.Rp), uv.reshape(H * L.vp, L.Rp)]), False, dev)
        return rows, self._out_columns(get(p + "o"), H, m.vdim, L.vp), None

    def _build_parallel(self, L, m: ParallelMixer, p: str, get):
        a, r, dev = m.left, m.right, self.dev
        self._attention_sizes(L, a)
        left, right = (lambda n: get(p + "left." + n)), (lambda n: get(p + "right." + n))
        L.dim, L.half, L.inv_freq, L.out_scale = a.dim, a.rot_dims // 2, self._angles(a.rot_base, a.rot_dims), m.left_scale
        L.q_w = head_rows(left("q.norm").float(), a.heads, a.dim, L.dp).contiguous()
        L.k_w = head_rows(left("k.norm").float(), a.kv_heads, a.dim, L.dp).contiguous()
        # state-space half: z | x | B | C | step sizes
        L.ssm, L.SH, L.SV, L.SG, L.norm_groups = True, r.heads, r.vdim, r.groups, r.norm_groups
        L.sv, L.Np = pad64(r.vdim), pad_up(r.state, F.SSD_STATE_SIZES)
        if L.Np not in F.SSD_STATE_SIZES:
            raise ValueError(f"the state-space mixer takes states of at most {F.SSD_STATE_SIZES[-1]} per head, got {r.state}")
        bc, wide = r.groups * r.state, L.SH * L.sv
        L.taps, L.C = r.taps, wide + 2 * r.groups * L.Np
        L.z_col = L.v_col + L.G * L.vp
        L.conv_col, L.dt_col = L.z_col + wide, L.z_col + wide + L.C

        def channels(t):
            """x, B and C with their heads and groups padded."""
            x, B, C = t.split([r.inner, bc, bc])
            return torch.cat([head_rows(x, r.heads, r.vdim, L.sv), head_rows(B, r.groups, r.state, L.Np), head_rows(C, r.groups, r.state, L.Np)])
        L.conv_w, L.conv_b = channels(right("conv")).t().float().contiguous(), channels(right("conv.b")).float().contiguous()
        L.dt_bias, L.D = right("dt_bias").float().contiguous(), right("D").float().contiguous()
        L.neg_a = -torch.exp(right("A_log").float()).contiguous()
        L.s_norm = head_rows(right("norm").float(), r.heads, r.vdim, L.sv).mul(m.right_scale).contiguous()
        z, xbc, dt = right("in").split([r.inner, r.conv_channels, r.heads])
        rows = torch.cat([self._qkv(L, a, left), head_rows(z, r.heads, r.vdim, L.sv), channels(xbc), pad_to(dt, pad8(r.heads), dt.shape[1])])
        L.n_left = L.heads * L.vp
        out = torch.cat([self._out_columns(left("o"), a.heads, a.vdim, L.vp), self._out_columns(right("o"), r.heads, r.vdim, L.sv)], 1)
        return rows, out, self._qkv(L, a, left, ".b")

    def weight_bytes(self, tokens: int = 1) -> int:
        """Bytes of weights a decode step of `tokens` tokens streams (experts: at most top per token and layer)."""
        n = self.head.nbytes()
        for L in self.layers:
            n += L.w_in.nbytes() + L.w_o.nbytes()
            if L.latent:
                n += (L.uk_t.numel() + L.uv.numel()) * L.uv.element_size()
            if L.moe is not None:
                n += self._expert_bytes(L, tokens)
            elif L.ff:
                n += L.w_up.nbytes() + L.w_down.nbytes()
        return n

    # ------------------------------------------------------------------ cache pages and state slots
    def _bytes_per_block(self) -> int:
        return sum(PAGE * (L.Rp if L.latent else L.G * (L.dp + L.vp)) for L in self.layers) * (4 if self.f32 else 2)

    def _state_bytes_per_slot(self) -> int:
        return sum(L.SH * L.Np * L.sv * 4 for L in self.ssm_layers) + sum((L.taps - 1) * L.C for L in self.attn_layers) * (4 if self.f32 else 2)

    def alloc_cache(self, num_blocks: int, block_size: int, num_slots: int):
        assert block_size == PAGE
        self.num_blocks = num_blocks
        new = lambda dt, *s: torch.zeros(*s, dtype=dt, device=self.dev)
        for L in self.layers:
            if L.latent:
                self.cache[L.index] = (new(self.dtype, num_blocks, PAGE, L.Rp),)
                continue
            self.cache[L.index] = (new(self.dtype, num_blocks, L.G, PAGE, L.dp), new(self.dtype, num_blocks, L.G, L.vp, PAGE))
            self.state[L.index, "conv"] = new(self.dtype, num_slots, L.taps - 1, L.C)
            if L.ssm:
                self.state[L.index, "ssm"] = new(torch.float32, num_slots, L.SH, L.Np, L.sv)

    # ------------------------------------------------------------------ step
    def _alloc_ctx(self, T: int, S: int, max_blocks: int, num_qg: int, nsplit: int) -> StepCtx:
        x, dev, dt, Ls = self._alloc_inputs(T, S, max_blocks, num_qg, nsplit), self.dev, self.dtype, self.layers
        # rows of padding sequences in a captured step are never written by the mixers: zeros, so that they stay finite
        new = torch.zeros if T <= 256 else torch.empty
        x.x = new(T, self.Wp, dtype=torch.float32, device=dev)
        x.h = new(T, self.Wp, dtype=dt, device=dev)
        x.proj = new(T * max(L.n_proj for L in Ls), dtype=dt, device=dev)
        x.mix = new(T * max(L.n_mix for L in Ls), dtype=dt, device=dev)
        dense = max((L.ff for L in Ls if L.moe is None), default=0)
        if dense:
            x.ff = new(T * dense, dtype=dt, device=dev)
        self._alloc_attention(x, T, num_qg, nsplit, self.attn_layers, new)
        if self.ssm_layers:
            x.xbc = new(T * max(L.C for L in self.ssm_layers), dtype=dt, device=dev)
            x.y = new(T * max(L.SH * L.sv for L in self.ssm_layers), dtype=torch.float32, device=dev)
        self._alloc_latent(x, T, num_qg, self.latent_layers, new)
        self._alloc_experts(x, T, [L for L in Ls if L.moe is not None], new)
        x.snaps, x.chunks, x.short, x.conv_tiles = [], {}, None, None      # chunks: chunk size -> (table, ranges); short: the other sequences
        return x

    def _prepare_step(self, x: StepCtx, batch):
        self._prepare_latent(x, batch, self.latent_layers)
        if self.attn_layers:
            x.conv_tiles = F.conv_tiles(batch.cu_seqlens).to(self.dev, non_blocking=True)
            self._prepare_recurrence(x, batch, [F.ssd_chunk_size(L.Np) for L in self.ssm_layers], self.ssd_chunk_min_tokens)

    def _latent_rows(self, L):
        return self.cache[L.index][0]

    def _conv_heads(self, L, x: StepCtx, proj):
        """Queries (returned), keys and values after their convolutions; keys and values into the cache pages."""
        m, (kc, vc), q = L.spec, self.cache[L.index], x.q[:x.T * L.heads * L.dp].view(x.T, L.heads * L.dp)
        p = self._conv_params(L, x, proj)
        p.positions, p.slot_mapping, p.q_out, p.kcache, p.vcache = ptr(x.positions), ptr(x.slot_mapping), ptr(q), ptr(kc), ptr(vc)
        p.H, p.G, p.dp, p.vp, p.num_blocks, p.temp_every, p.temp_coef = L.heads, L.G, L.dp, L.vp, self.num_blocks, m.temp_every, m.temp_coef
        F.conv(p, self.f32)
        self._launches += 1 + (x.cu is not None and L.taps > 1)
        return q

    def _normed_heads(self, L, x: StepCtx, proj):
        """Normed and turned queries (returned) and keys; keys and values into the cache pages."""
        (kc, vc), q = self.cache[L.index], x.q[:x.T * L.heads * L.dp].view(x.T, L.heads * L.dp)
        r = NormRopeParams()
        r.proj, r.q_w, r.k_w, r.inv_freq, r.positions, r.slot_mapping = (ptr(t) for t in (proj, L.q_w, L.k_w, L.inv_freq, x.positions, x.slot_mapping))
        r.q_out, r.kcache, r.vcache = ptr(q), ptr(kc), ptr(vc)
        r.T, r.ld, r.q_col, r.k_col, r.v_col, r.H, r.G = x.T, proj.stride(0), 0, L.k_col, L.v_col, L.heads, L.G
        r.dim, r.dp, r.vp, r.half, r.num_blocks, r.eps = L.dim, L.dp, L.vp, L.half, self.num_blocks, self.cfg.rms_eps
        F.norm_rope(r, self.f32)
        self._launches += 1
        return q

    def _ssd_params(self, L, x: StepCtx, xbc, proj, mix) -> SsdParams:
        p, wide = SsdParams(), L.SH * L.sv
        p.xbc, p.proj, p.dt_bias, p.neg_a, p.D, p.norm = ptr(xbc), ptr(proj), ptr(L.dt_bias), ptr(L.neg_a), ptr(L.D), ptr(L.s_norm)
        p.state, p.slots, p.cu, p.y, p.out = ptr(self.state[L.index, "ssm"]), ptr(x.slots), ptr(x.cu), ptr(x.y), ptr(mix[:, L.n_left:])
        if x.snaps:
            p.snap_rel, p.snap_idx, p.snap, p.num_snap = ptr(x.snap_rel), ptr(x.snap_idx), ptr(x.snap_state[L.index, "ssm"]), x.num_snap
        p.ldx, p.ld, p.ldo, p.x_col, p.b_col, p.c_col = L.C, proj.stride(0), mix.stride(0), 0, wide, wide + L.SG * L.Np
        p.z_col, p.dt_col, p.H, p.G, p.V, p.vp, p.norm_groups, p.eps = L.z_col, L.dt_col, L.SH, L.SG, L.SV, L.sv, L.norm_groups, self.cfg.rms_eps
        if x.short is not None:
            ck, rng = x.chunks[F.ssd_chunk_size(L.Np)]
            p.ck_seq, p.ck_tok0, p.ck_ntok, p.ck_snap = (ptr(r) for r in ck)
            p.long_seq, p.long_ck, p.nc, p.num_long = ptr(x.longs), ptr(rng), ck.shape[1], x.longs.numel()
            p.g_ws, p.s_ws = (ptr(w) for w in self.ssd_ws.get(p.nc, L.SH, L.Np, L.sv))
            p.seqs = ptr(x.short)
        return p

    def _state_space(self, L, x: StepCtx, proj, mix):
        p = self._ssd_params(L, x, self._conv_inputs(L, x, proj), proj, mix)
        if x.short is not None:
            F.ssd_chunked(p, L.Np)
            self._launches += 3
        num = x.S if x.short is None else x.short.numel()
        if num:
            F.ssd_step(p, num, L.Np, self.f32)
        F.ssd_finish(p, x.T, self.f32)
        self._launches += 1 + bool(num)

    def _mixer(self, L, x: StepCtx, proj, mix):
        if L.latent:
            F.latent_rope(proj, L.heads, L.dp, L.dim, L.kv_col, L.kv_norm, L.inv_freq, x.positions, x.slot_mapping, self._latent_rows(L), L.R,
                          self.cfg.rms_eps)
            self._launches += 1
            if x.num_qg:
                self._attn_latent_short(L, x, proj, mix)
            if x.reach:
                self._attn_latent_long(L, x, proj, mix)        # after the split attention, whose row range may span these
        elif L.ssm:
            self._attention(L, x, self._normed_heads(L, x, proj), proj, mix)
            self._state_space(L, x, proj, mix)
        else:
            self._attention(L, x, self._conv_heads(L, x, proj), proj, mix)

    def _run_layers(self, x: StepCtx):
        c, T = self.cfg, x.T
        F.embed_pos(x.ids, x.positions, self.embed, None, None, x.x, self.W, c.rms_eps)
        F.rmsnorm_f32(x.x, self.layers[0].norm1, x.h, self.W, c.rms_eps)
        self._launches += 2
        into_x = lambda bias=None: F.gemm_epilogue(resid32=x.x, bias=bias)
        for i, L in enumerate(self.layers):
            nvtx_mark(f"layer {i}")
            proj, mix = x.proj[:T * L.n_proj].view(T, L.n_proj), x.mix[:T * L.n_mix].view(T, L.n_mix)
            n = L.w_in(x.h, proj, F.GEPI_STORE, None if L.in_bias is None else F.gemm_epilogue(bias=L.in_bias))
            self._mixer(L, x, proj, mix)
            n += L.w_o(mix, x.x, F.GEPI_RESID32, into_x())
            after = self.layers[i + 1].norm1 if i + 1 < len(self.layers) else None
            if L.moe is not None:
                g, rows = self._norm_and_route(L, x, None, None)
                self._experts(L, x, g, rows)
                F.resid_norm(rows, x.x, None, x.h, after, self.W, c.rms_eps, routed=g)
                n += 1
            else:
                if L.ff:
                    act = x.ff[:T * L.ff].view(T, L.ff)
                    F.rmsnorm_f32(x.x, L.norm2, x.h, self.W, c.rms_eps)
                    n += 1 + L.w_up(x.h, act, F.GEPI_SPLIT_GLU, F.gemm_epilogue(out2=act, n_split=0, glu=SILU_UNIT, bias=L.up_bias))
                    n += L.w_down(act, x.x, F.GEPI_RESID32, into_x(L.down_bias))
                if after is not None:
                    F.rmsnorm_f32(x.x, after, x.h, self.W, c.rms_eps)
                    n += 1
            self._launches += n
        nvtx_end()
        return x.x

    def _lm_head(self, hidden, logits, n):
        h = torch.empty(n, self.Wp, dtype=self.dtype, device=self.dev)
        F.rmsnorm_f32(hidden, self.final_norm, h, self.W, self.cfg.rms_eps)
        self._launches += 1 + self.head(h, logits, F.GEPI_F32, F.gemm_epilogue(softcap=self.cfg.logit_softcap))

    def _status_ptr(self) -> int:
        return self.status
