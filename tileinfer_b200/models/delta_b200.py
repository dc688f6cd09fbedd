"""Luvapel on one B200: weights in kernel layout, pages of keys and values, slots of recurrent states and convolution tails,
the fused step.

Per layer a decode step launches

  input product -> parallel:       head norms + rotation + cache store -> paged attention [window, gate] (+ merge), and
                                   convolutions + silu -> state step -> head norm + gate
                   general_delta:  state step [decay's second product, rates, unit keys] -> head norm + gate
  -> output product(s) -> [branch norms, gate, norm, residual add, next input]
  -> up product [square of the positive part in the epilogue] -> down product -> [gate, norm, residual add, next input]

The logits of the residual's gates are columns of the input product and of the up product, which read the same rows.  The
values of an attention layer are its key columns, and a head's temperature is part of its query weights.  Long portions of
prompts run the tcgen05 attention over the paged cache and the chunked form of the delta rules.  Head sizes are padded with
zero weights, so any size runs.  A layer that reuses another one's tensors has a cache and state of its own.  quant: "bf16",
"w8a16" (int8 projections) or "fp32" (everything in 32 bits).  The residual, norms, angles, attention scores, decays, rates and
states are fp32 in every mode.
"""
from __future__ import annotations

import copy

import torch

from ..ops import functional as F
from ..ops.functional import DeltaParams, RopeUnitParams, ptr
from ..utils.trace import nvtx_end, nvtx_mark
from .attention_b200 import AttentionLayers, head_rows, pad8, pad_up
from .conv_b200 import ConvLayers
from .luvapel import BRANCH_SCALE, DECAY_SCALE, GeneralDelta, LuvapelConfig, ParallelMixer
from .paged_state_b200 import PAGE, PagedState
from .products_b200 import Product, pad64, pad_to
from .runtime_b200 import DeviceRuntime, StepCtx


class _Layer:
    attn = False                         # keys and values in pages
    n_left = ff = 0                      # columns of the attention's output; feed-forward


class B200DeltaModel(PagedState, AttentionLayers, ConvLayers, DeviceRuntime):
    def __init__(self, cfg: LuvapelConfig, src, *, quant="bf16", tp=1, rank=0, comm=None, config=None):
        assert torch.cuda.is_available(), "B200DeltaModel needs a CUDA device"
        cfg.validate_tp(tp)
        # load (or build) the kernel libraries the layers need now: fail loudly
        F.L("base", "rows", "delta", *(["attention", "conv"] if cfg.num_attn_layers else []))
        self.cfg, self.tp, self.rank, self.comm, self.peer = cfg, tp, rank, comm, None
        self.dev = torch.device("cuda", torch.cuda.current_device())
        self.quant, self.f32 = quant, quant == "fp32"
        self.dtype = torch.float32 if self.f32 else torch.bfloat16
        self.W, self.Wp = cfg.hidden_size, pad64(cfg.hidden_size)
        self.vocab_start, self.v_local = 0, cfg.vocab_size
        self._build(src)
        torch.cuda.empty_cache()
        self.attn_layers = [L for L in self.layers if L.attn]
        self.hkv = max((L.G * L.rep for L in self.attn_layers), default=1)            # blocks per query group of the split attention
        # heads wider than the tensor-core kernels take: every token of every layer is a query of the split forms
        tiled = not self.f32 and all(L.dp <= 256 for L in self.attn_layers)
        self.PREFILL_ATTN_MIN_TOKENS = 32 if tiled else 1 << 30
        # sequences with at least this many tokens in a step run the recurrences in chunks
        chunked = not self.f32 and all(F.delta_chunk_size(L.dk) for L in self.layers)
        self.delta_chunk_min_tokens = 32 if chunked else 1 << 30
        self.delta_ws = F.DeltaWorkspace(self.dev)
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
        self.final_norm = self._vec(get("final.norm"), Wp)
        own = {i: self._build_layer(spec, f"l{i}.", get) for i, spec in enumerate(c.layers) if spec.weights_of is None}
        self.layers = [copy.copy(own[c.owner(i)]) for i in range(c.num_layers)]
        for i, L in enumerate(self.layers):
            L.index = i
        self.head = Product(pad_to(get("head"), c.vocab_size, Wp), "fp32" if self.f32 else "bf16", dev)

    def _product(self, w: torch.Tensor) -> Product:
        return Product(w, self.quant, self.dev)

    def _build_layer(self, spec, p: str, get) -> _Layer:
        L, Wp = _Layer(), self.Wp
        L.spec, L.parallel, L.norm1 = spec.mixer, isinstance(spec.mixer, ParallelMixer), self._vec(get(p + "norm1"), Wp)
        rows = (self._build_parallel if L.parallel else self._build_general)(L, spec.mixer, p + "mix.", get)
        n = sum(r.shape[0] for r in rows)
        L.w_in = self._product(torch.cat([pad_to(r, r.shape[0], Wp) for r in rows] + [pad_to(get(p + "rg1"), Wp, Wp)]))
        L.n_proj, L.rg_col = L.w_in.N, n
        L.in_bias = torch.cat([torch.zeros(n, device=self.dev), self._vec(get(p + "rg1.b"), Wp)])
        if spec.mlp is not None:
            L.norm2, L.ff = self._vec(get(p + "norm2"), Wp), pad64(spec.mlp.ff)
            L.w_up = self._product(torch.cat([pad_to(get(p + "rg2"), Wp, Wp), pad_to(get(p + "mlp.up"), L.ff, Wp)]))
            L.up_bias = torch.cat([self._vec(get(p + "rg2.b"), Wp), torch.zeros(L.ff, device=self.dev)])
            L.w_down = self._product(pad_to(get(p + "mlp.down"), Wp, L.ff))
        return L

    def _delta_sizes(self, L, heads: int, kv_heads: int, dim: int, vdim: int, col: int):
        """Heads, padded sizes, and the columns of queries, keys and values from `col` on.  Returns their end."""
        L.DH, L.rep_d, L.dk, L.dv, L.vdim = heads, heads // kv_heads, pad_up(dim, F.GLA_KEY_SIZES), pad64(vdim), vdim
        if L.dk not in F.GLA_KEY_SIZES:
            raise ValueError(f"a delta rule takes keys of at most {F.GLA_KEY_SIZES[-1]} per head, got {dim}")
        L.n_right = heads * L.dv
        L.dq_col, L.dk_col, L.dv_col = col, col + kv_heads * L.dk, col + 2 * kv_heads * L.dk
        return L.dv_col + heads * L.dv

    def _build_parallel(self, L, m: ParallelMixer, p: str, get) -> list:
        a, r, Wp = m.left, m.right, self.Wp
        left, right = (lambda n: get(p + "left." + n)), (lambda n: get(p + "right." + n))
        self._attention_sizes(L, a)
        L.v_col, L.n_left = L.k_col, a.heads * L.vp           # the values are the keys as projected
        L.gate_col = L.k_col + L.G * L.dp
        L.inv_freq, L.half = self._angles(a.rot_base, a.rot_dims), a.rot_dims // 2
        temp = left("temp").float()
        L.q_w = pad_to(temp[:, None] * left("q.norm").float()[None], a.heads, L.dp).flatten().contiguous()
        L.k_w = pad_to(left("k.norm").float()[None].expand(a.kv_heads, -1), a.kv_heads, L.dp).flatten().contiguous()
        # gated delta rule: channels of the convolution | gate | steps | decays
        L.conv_col, L.taps = L.gate_col + L.n_left, r.taps
        end = self._delta_sizes(L, r.heads, r.kv_heads, r.dim, r.vdim, 0)
        L.C = end
        channels = lambda s: torch.cat([head_rows(right("q" + s), r.kv_heads, r.dim, L.dk), head_rows(right("k" + s), r.kv_heads, r.dim, L.dk),
                                        head_rows(right("v" + s), r.heads, r.vdim, L.dv)])
        L.conv_w, L.conv_b = channels(".conv").t().float().contiguous(), None
        L.dgate_col = L.conv_col + L.C
        L.b_col = L.dgate_col + L.n_right
        L.a_col = L.b_col + pad8(r.heads)
        L.d_bias, L.neg_a = right("dt_bias").float().contiguous(), -torch.exp(right("A_log").float()).contiguous()
        L.R, L.q_scale, L.h_norm = 0, r.dim ** -0.5, self._vec(right("norm"), L.dv)
        L.left_out, L.right_out = self._vec(left("out"), Wp), self._vec(right("out"), Wp)
        out = lambda w, H, n, np_: self._product(pad_to(self._out_columns(w, H, n, np_), Wp, H * np_))
        L.w_o, L.w_o2 = out(left("o"), a.heads, a.vdim, L.vp), out(right("o"), r.heads, r.vdim, L.dv)
        few = lambda w: pad_to(w, pad8(r.heads), w.shape[1])
        return [head_rows(left("q"), a.heads, a.dim, L.dp), head_rows(left("k"), a.kv_heads, a.dim, L.dp), head_rows(left("g"), a.heads, a.vdim, L.vp),
                channels(""), head_rows(right("g"), r.heads, r.vdim, L.dv), few(right("b")), few(right("a"))]

    def _build_general(self, L, m: GeneralDelta, p: str, get) -> list:
        H, n = m.heads, m.dim
        L.dgate_col = self._delta_sizes(L, H, H, n, n, 0)
        L.b_col = L.dgate_col + L.n_right
        L.a_col, L.R, L.q_scale, L.neg_a = L.b_col + H * L.dk, m.decay_rank, 1.0, None
        keyed = lambda t: pad_to(t.float().view(H, n), H, L.dk).flatten().contiguous()
        L.d_bias, L.w0 = keyed(get(p + "a.b")), keyed(get(p + "w0"))
        L.w2 = head_rows(get(p + "w2"), H, n, L.dk).t().float().contiguous()
        L.h_norm = pad_to(get(p + "norm").float().view(H, n), H, L.dv).contiguous()
        L.w_o = self._product(pad_to(self._out_columns(get(p + "o"), H, n, L.dv), self.Wp, L.n_right))
        head = lambda t, to: head_rows(get(p + t), H, n, to)
        w1 = get(p + "w1")
        return [head("r", L.dk), head("k", L.dk), head("v", L.dv), head("g", L.dv), head("a", L.dk), pad_to(w1, pad8(L.R), w1.shape[1])]

    def weight_bytes(self, tokens: int = 1) -> int:
        """Bytes of weights a decode step streams."""
        n = self.head.nbytes()
        for L in self.layers:
            n += L.w_in.nbytes() + L.w_o.nbytes() + (L.w_o2.nbytes() if L.parallel else 0)
            n += L.w_up.nbytes() + L.w_down.nbytes() if L.ff else 0
        return n

    # ------------------------------------------------------------------ cache pages and state slots
    def _bytes_per_block(self) -> int:
        return sum(PAGE * L.G * (L.dp + L.vp) for L in self.attn_layers) * (4 if self.f32 else 2)

    def _state_bytes_per_slot(self) -> int:
        return sum(L.DH * L.dk * L.dv * 4 for L in self.layers) + sum((L.taps - 1) * L.C for L in self.attn_layers) * (4 if self.f32 else 2)

    def alloc_cache(self, num_blocks: int, block_size: int, num_slots: int):
        assert block_size == PAGE
        self.num_blocks = num_blocks
        new = lambda dt, *s: torch.zeros(*s, dtype=dt, device=self.dev)
        for L in self.layers:
            if L.attn:
                self.cache[L.index] = (new(self.dtype, num_blocks, L.G, PAGE, L.dp), new(self.dtype, num_blocks, L.G, L.vp, PAGE))
                self.state[L.index, "conv"] = new(self.dtype, num_slots, L.taps - 1, L.C)
            self.state[L.index, "delta"] = new(torch.float32, num_slots, L.DH, L.dk, L.dv)

    # ------------------------------------------------------------------ step
    def _alloc_ctx(self, T: int, S: int, max_blocks: int, num_qg: int, nsplit: int) -> StepCtx:
        x, dev, dt, Ls = self._alloc_inputs(T, S, max_blocks, num_qg, nsplit), self.dev, self.dtype, self.layers
        # rows of padding sequences in a captured step are never written by the mixers: zeros, so that they stay finite
        new = torch.zeros if T <= 256 else torch.empty
        x.x = new(T, self.Wp, dtype=torch.float32, device=dev)
        x.h, x.y, x.y2, x.gate = (new(T, self.Wp, dtype=dt, device=dev) for _ in range(4))
        x.proj = new(T * max(L.n_proj for L in Ls), dtype=dt, device=dev)
        x.left = new(T * max(max(L.n_left for L in Ls), 1), dtype=dt, device=dev)
        x.right = new(T * max(L.n_right for L in Ls), dtype=dt, device=dev)
        x.o = new(T * max(L.n_right for L in Ls), dtype=torch.float32, device=dev)
        x.ff = new(T * max(max(L.ff for L in Ls), 1), dtype=dt, device=dev)
        if self.attn_layers:
            x.xbc = new(T * max(L.C for L in self.attn_layers), dtype=dt, device=dev)
        self._alloc_attention(x, T, num_qg, nsplit, self.attn_layers, new)
        x.snaps, x.chunks, x.short, x.conv_tiles = [], {}, None, None      # chunks: chunk size -> (table, ranges); short: the other sequences
        return x

    def _prepare_step(self, x: StepCtx, batch):
        if self.attn_layers:
            x.conv_tiles = F.conv_tiles(batch.cu_seqlens).to(self.dev, non_blocking=True)
        self._prepare_recurrence(x, batch, [F.delta_chunk_size(L.dk) for L in self.layers], self.delta_chunk_min_tokens)

    def _rotate_and_store(self, L, x: StepCtx, proj):
        """Normed and turned queries (returned) and keys, and the keys as projected as values; keys and values into the cache pages."""
        (kc, vc), q = self.cache[L.index], x.q[:x.T * L.heads * L.dp].view(x.T, L.heads * L.dp)
        r = RopeUnitParams()
        r.proj, r.inv_freq, r.positions, r.slot_mapping = ptr(proj), ptr(L.inv_freq), ptr(x.positions), ptr(x.slot_mapping)
        r.q_out, r.kcache, r.vcache, r.status, r.q_w, r.k_w = ptr(q), ptr(kc), ptr(vc), self.status, ptr(L.q_w), ptr(L.k_w)
        r.T, r.ld, r.q_col, r.k_col, r.v_col, r.H, r.G = x.T, proj.stride(0), 0, L.k_col, L.v_col, L.heads, L.G
        r.dim, r.dp, r.vp, r.half, r.num_blocks, r.eps, r.pairs = L.spec.left.dim, L.dp, L.vp, L.half, self.num_blocks, self.cfg.rms_eps, 1
        F.rope_unit(r, self.f32)
        self._launches += 1
        return q

    def _delta_params(self, L, x: StepCtx, src, proj) -> DeltaParams:
        p = DeltaParams()
        p.src, p.proj, p.bias, p.neg_a, p.state, p.slots = ptr(src), ptr(proj), ptr(L.d_bias), ptr(L.neg_a), ptr(self.state[L.index, "delta"]), ptr(x.slots)
        if not L.parallel:
            p.w2, p.w0, p.decay_scale = ptr(L.w2), ptr(L.w0), DECAY_SCALE
        p.cu, p.o = ptr(x.cu), ptr(x.o)
        if x.snaps:
            p.snap_rel, p.snap_idx, p.snap, p.num_snap = ptr(x.snap_rel), ptr(x.snap_idx), ptr(x.snap_state[L.index, "delta"]), x.num_snap
        p.lds, p.ld, p.H, p.rep, p.R = src.stride(0), proj.stride(0), L.DH, L.rep_d, L.R
        p.q_col, p.k_col, p.v_col, p.b_col, p.a_col, p.q_scale = L.dq_col, L.dk_col, L.dv_col, L.b_col, L.a_col, L.q_scale
        return p

    def _delta(self, L, x: StepCtx, proj, out):
        """The layer's delta rule over the step's tokens; gated heads into `out`."""
        p = self._delta_params(L, x, self._conv_inputs(L, x, proj) if L.parallel else proj, proj)
        if x.short is not None:
            ck, rng = x.chunks[F.delta_chunk_size(L.dk)]
            p.ck_seq, p.ck_tok0, p.ck_ntok, p.ck_snap = (ptr(r) for r in ck)
            p.long_seq, p.long_ck, p.nc, p.num_long = ptr(x.longs), ptr(rng), ck.shape[1], x.longs.numel()
            p.t_ws, p.q_ws, p.s_ws, p.f_ws = (ptr(w) for w in self.delta_ws.get(p.nc, L.DH, L.dk, L.dv))
            F.delta_chunked(p, L.dk, L.dv, not L.parallel)
            p.seqs = ptr(x.short)
            self._launches += 3
        num = x.S if x.short is None else x.short.numel()
        if num:
            F.delta_step(p, num, L.dk, L.dv, not L.parallel, self.f32)
        o = x.o[:x.T * L.n_right].view(x.T, L.DH, L.dv)
        F.head_norm(o, proj, L.dgate_col, L.h_norm, out, L.vdim, self.cfg.rms_eps, silu=L.parallel)
        self._launches += 1 + bool(num)

    def _run_layers(self, x: StepCtx):
        c, T, W = self.cfg, x.T, self.W
        F.embed_pos(x.ids, x.positions, self.embed, None, None, x.x, W, c.rms_eps, scale=c.embedding_scale, h=x.h)
        self._launches += 1
        for i, L in enumerate(self.layers):
            nvtx_mark(f"layer {i}")
            proj, right = x.proj[:T * L.n_proj].view(T, L.n_proj), x.right[:T * L.n_right].view(T, L.n_right)
            n = L.w_in(x.h, proj, F.GEPI_STORE, F.gemm_epilogue(bias=L.in_bias))
            if L.parallel:
                left = x.left[:T * L.n_left].view(T, L.n_left)
                self._attention(L, x, self._rotate_and_store(L, x, proj), proj, left)
                self._delta(L, x, proj, right)
                n += L.w_o(left, x.y, F.GEPI_STORE) + L.w_o2(right, x.y2, F.GEPI_STORE)
                F.gated_norm(x.y, proj[:, L.rg_col:], x.x, L.norm1, x.h, W, c.rms_eps, y2=x.y2, w_y=L.left_out, w_y2=L.right_out, scale=BRANCH_SCALE)
            else:
                self._delta(L, x, proj, right)
                n += L.w_o(right, x.y, F.GEPI_STORE)
                F.gated_norm(x.y, proj[:, L.rg_col:], x.x, L.norm1, x.h, W, c.rms_eps)
            if L.ff:
                act = x.ff[:T * L.ff].view(T, L.ff)
                n += L.w_up(x.h, x.gate, F.GEPI_SPLIT_RELU2, F.gemm_epilogue(out2=act, n_split=self.Wp, bias=L.up_bias))
                n += L.w_down(act, x.y, F.GEPI_STORE)
                F.gated_norm(x.y, x.gate, x.x, L.norm2, x.h, W, c.rms_eps)
                n += 1
            self._launches += n + 1
        nvtx_end()
        return x.x

    def _lm_head(self, hidden, logits, n):
        h = torch.empty(n, self.Wp, dtype=self.dtype, device=self.dev)
        F.rmsnorm_f32(hidden, self.final_norm, h, self.W, self.cfg.rms_eps)
        self._launches += 1 + self.head(h, logits, F.GEPI_F32)

    def _status_ptr(self) -> int:
        return self.status
