"""Tensor-level wrappers of the sm_100a kernels (torch tensors in, launches on the current stream).

Nothing here allocates unless the docstring says so; the model keeps its activations, workspaces and
parameter blocks alive, which also makes every launch capturable into a CUDA graph.
"""
from __future__ import annotations

import ctypes
import math
import os

import torch

from . import lib as _l
from .lib import ChainParams, GemvParams, MAX_CHAIN, MAX_RANKS, check, ptr, stream

_I, _P, _F, _LL = ctypes.c_int, ctypes.c_void_p, ctypes.c_float, ctypes.c_longlong

XGLOBAL, XNORM = 0, 1
EPI_STORE, EPI_SWIGLU, EPI_ROWPAR, EPI_F32, EPI_ARGMAX = 0, 1, 2, 3, 4
W_INT8, W_BF16 = 0, 1


def _device_sm_count() -> int:
    """Streaming multiprocessors of the current GPU (148 on a B200; the fallback when no GPU is visible).  The
    persistent GEMV launches one CTA per SM and its grid barrier needs every CTA resident, so the grid must follow
    the device, not a constant."""
    try:
        if torch.cuda.is_available():
            return int(torch.cuda.get_device_properties(torch.cuda.current_device()).multi_processor_count)
    except Exception:
        pass
    return 148


NUM_SMS = _device_sm_count()
GEMV_WARPS = int(os.environ.get("TI_GEMV_WARPS", "16"))   # must match the -DTI_GEMV_WARPS the library was built with
GEMV_TPS = int(os.environ.get("TI_GEMV_TPS", "8"))            # 512-byte tiles per ring stage
GEMV_MAX_STAGES = int(os.environ.get("TI_GEMV_STAGES", "6"))
GEMV_UNITS_PER_WARP = int(os.environ.get("TI_GEMV_UPW", "4"))


class GdnParams(ctypes.Structure):
    _fields_ = [("proj", _P), ("conv_w", _P), ("neg_a_exp", _P), ("dt_bias", _P), ("norm_w", _P), ("state", _P),
                ("conv_state", _P), ("slots", _P), ("cu", _P), ("out", _P), ("snap_rel", _P), ("snap_state", _P),
                ("snap_conv", _P), ("ld", _I), ("hk", _I), ("hv", _I), ("num_snap", _I), ("eps", _F), ("snap_idx", _P), ("status", _P)]


class GdnChunkParams(ctypes.Structure):
    _fields_ = [("proj", _P), ("conv_w", _P), ("neg_a_exp", _P), ("dt_bias", _P), ("norm_w", _P), ("state", _P),
                ("conv_state", _P), ("slots", _P), ("cu", _P), ("out", _P), ("snap_rel", _P), ("snap_idx", _P),
                ("snap_state", _P), ("snap_conv", _P), ("ck_seq", _P), ("ck_tok0", _P), ("ck_ntok", _P), ("ck_snap", _P),
                ("seq_ck", _P), ("wf", _P), ("qf", _P), ("mf", _P), ("kf", _P), ("u", _P), ("gamma", _P),
                ("ld", _I), ("hk", _I), ("hv", _I), ("num_snap", _I), ("nc", _I), ("eps", _F)]


class QkvPrepParams(ctypes.Structure):
    _fields_ = [("proj", _P), ("q_norm", _P), ("k_norm", _P), ("positions", _P), ("slot_mapping", _P),
                ("q_out", _P), ("kcache", _P), ("vcache", _P), ("ld", _I), ("hq", _I), ("hkv", _I),
                ("rotary_dim", _I), ("eps", _F), ("log2_theta", _F), ("num_blocks", _I), ("status", _P)]


class AttnParams(ctypes.Structure):
    _fields_ = [("q", _P), ("kcache", _P), ("vcache", _P), ("block_tables", _P), ("positions", _P),
                ("qg_seq", _P), ("qg_tok0", _P), ("qg_ntok", _P), ("o_part", _P), ("ml_part", _P),
                ("gate_src", _P), ("out", _P), ("hq", _I), ("hkv", _I), ("max_blocks", _I), ("nsplit", _I),
                ("ld", _I), ("num_qg", _I), ("scale_log2e", _F), ("num_blocks", _I), ("status", _P), ("cap_in", _F), ("cap_out", _F),
                ("rep", _I), ("window", _I), ("slopes", _P), ("head_gate", _P), ("ldg", _I), ("gcol", _I), ("ldo", _I), ("out_scale", _F), ("gate_col", _I), ("gate_stride", _I)]

    def __init__(self, *args, **kw):
        super().__init__(*args, **kw)
        self.out_scale = kw.get("out_scale", 1.0)


class LatentAttnParams(ctypes.Structure):
    _fields_ = [("q", _P), ("cache", _P), ("block_tables", _P), ("positions", _P), ("qg_seq", _P), ("qg_tok0", _P),
                ("qg_ntok", _P), ("sink", _P), ("o_part", _P), ("ml_part", _P), ("out", _P), ("status", _P),
                ("H", _I), ("R", _I), ("Rp", _I), ("max_blocks", _I), ("nsplit", _I), ("num_qg", _I), ("window", _I),
                ("num_blocks", _I), ("scale", _F), ("Ro", _I)]


class RopeUnitParams(ctypes.Structure):
    _fields_ = [("proj", _P), ("inv_freq", _P), ("positions", _P), ("slot_mapping", _P), ("q_out", _P), ("kcache", _P), ("vcache", _P),
                ("status", _P), ("T", _I), ("ld", _I), ("q_col", _I), ("k_col", _I), ("v_col", _I), ("H", _I), ("G", _I), ("dim", _I),
                ("dp", _I), ("vp", _I), ("half", _I), ("num_blocks", _I), ("eps", _F), ("pairs", _I), ("q_w", _P), ("k_w", _P)]


class AttnGeneralParams(ctypes.Structure):
    _fields_ = [("q", _P), ("kcache", _P), ("vcache", _P), ("block_tables", _P), ("positions", _P), ("qg_seq", _P), ("qg_tok0", _P),
                ("qg_ntok", _P), ("out", _P), ("status", _P), ("H", _I), ("G", _I), ("dp", _I), ("vp", _I), ("max_blocks", _I),
                ("num_qg", _I), ("num_blocks", _I), ("ldo", _I), ("scale", _F), ("softcap", _F), ("window", _I), ("slopes", _P),
                ("head_gate", _P), ("ldg", _I), ("gcol", _I), ("out_scale", _F), ("gate", _P)]

    def __init__(self, *args, **kw):
        super().__init__(*args, **kw)
        self.out_scale = kw.get("out_scale", 1.0)


class GlaParams(ctypes.Structure):
    _fields_ = [("proj", _P), ("a2", _P), ("a2_bias", _P), ("norm", _P), ("state", _P), ("slots", _P), ("cu", _P), ("seqs", _P),
                ("o", _P), ("out", _P), ("snap_rel", _P), ("snap_idx", _P), ("snap", _P),
                ("ld", _I), ("ldo", _I), ("H", _I), ("R", _I), ("q_col", _I), ("k_col", _I), ("v_col", _I), ("g_col", _I), ("a_col", _I),
                ("num_snap", _I), ("vdim", _I), ("q_scale", _F), ("inv_tau", _F), ("eps", _F),
                ("ck_seq", _P), ("ck_tok0", _P), ("ck_ntok", _P), ("ck_snap", _P), ("long_seq", _P), ("long_ck", _P), ("g_ws", _P),
                ("s_ws", _P), ("nc", _I), ("num_long", _I)]


class NormRopeParams(ctypes.Structure):
    _fields_ = [("proj", _P), ("q_w", _P), ("k_w", _P), ("inv_freq", _P), ("positions", _P), ("slot_mapping", _P), ("q_out", _P),
                ("kcache", _P), ("vcache", _P), ("T", _I), ("ld", _I), ("q_col", _I), ("k_col", _I), ("v_col", _I), ("H", _I), ("G", _I),
                ("dim", _I), ("dp", _I), ("vp", _I), ("half", _I), ("num_blocks", _I), ("eps", _F)]


class ConvParams(ctypes.Structure):
    _fields_ = [("proj", _P), ("w", _P), ("bias", _P), ("state", _P), ("slots", _P), ("cu", _P), ("tiles", _P), ("out", _P),
                ("positions", _P), ("slot_mapping", _P), ("q_out", _P), ("kcache", _P), ("vcache", _P), ("snap_rel", _P), ("snap_idx", _P),
                ("snap", _P), ("T", _I), ("S", _I), ("ld", _I), ("col", _I), ("C", _I), ("taps", _I), ("num_tiles", _I), ("ldo", _I),
                ("silu", _I), ("H", _I), ("G", _I), ("dp", _I), ("vp", _I), ("num_blocks", _I), ("temp_every", _I), ("num_snap", _I),
                ("temp_coef", _F)]


class SsdParams(ctypes.Structure):
    _fields_ = [("xbc", _P), ("proj", _P), ("dt_bias", _P), ("neg_a", _P), ("D", _P), ("norm", _P), ("state", _P), ("slots", _P),
                ("cu", _P), ("seqs", _P), ("y", _P), ("out", _P), ("snap_rel", _P), ("snap_idx", _P), ("snap", _P),
                ("ldx", _I), ("ld", _I), ("ldo", _I), ("x_col", _I), ("b_col", _I), ("c_col", _I), ("z_col", _I), ("dt_col", _I),
                ("H", _I), ("G", _I), ("V", _I), ("vp", _I), ("num_snap", _I), ("norm_groups", _I), ("eps", _F),
                ("ck_seq", _P), ("ck_tok0", _P), ("ck_ntok", _P), ("ck_snap", _P), ("long_seq", _P), ("long_ck", _P), ("g_ws", _P),
                ("s_ws", _P), ("nc", _I), ("num_long", _I)]


class DeltaParams(ctypes.Structure):
    _fields_ = [("src", _P), ("proj", _P), ("bias", _P), ("neg_a", _P), ("w2", _P), ("w0", _P), ("state", _P), ("slots", _P), ("cu", _P),
                ("seqs", _P), ("o", _P), ("snap_rel", _P), ("snap_idx", _P), ("snap", _P),
                ("lds", _I), ("ld", _I), ("H", _I), ("rep", _I), ("R", _I), ("q_col", _I), ("k_col", _I), ("v_col", _I), ("b_col", _I),
                ("a_col", _I), ("num_snap", _I), ("q_scale", _F), ("decay_scale", _F),
                ("ck_seq", _P), ("ck_tok0", _P), ("ck_ntok", _P), ("ck_snap", _P), ("long_seq", _P), ("long_ck", _P), ("t_ws", _P),
                ("q_ws", _P), ("s_ws", _P), ("f_ws", _P), ("nc", _I), ("num_long", _I)]


class HeadNormParams(ctypes.Structure):
    _fields_ = [("o", _P), ("gate", _P), ("norm", _P), ("out", _P), ("ld", _I), ("ldo", _I), ("g_col", _I), ("H", _I), ("dv", _I),
                ("vdim", _I), ("norm_stride", _I), ("silu", _I), ("eps", _F)]


class GatedNormParams(ctypes.Structure):
    _fields_ = [("y", _P), ("y2", _P), ("gate", _P), ("w_y", _P), ("w_y2", _P), ("w_out", _P), ("x", _P), ("h", _P),
                ("W", _I), ("P", _I), ("ldy", _I), ("ldg", _I), ("eps", _F), ("scale", _F)]


class MoeRouteParams(ctypes.Structure):
    _fields_ = [("logits", _P), ("correction", _P), ("valid", _P), ("ids", _P), ("weight", _P), ("pos", _P), ("counts", _P),
                ("ticket", _P), ("first", _P), ("tiles", _P), ("num_tiles", _P), ("M", _I), ("E", _I), ("identity", _I), ("top", _I),
                ("groups", _I), ("keep", _I), ("ldl", _I), ("tile_rows", _I), ("max_tiles", _I), ("row_stride", _I)]


class ResidNormParams(ctypes.Structure):
    _fields_ = [("y", _P), ("x", _P), ("w_out", _P), ("w_next", _P), ("h", _P), ("slot", _P), ("weight", _P), ("h_in", _P),
                ("W", _I), ("P", _I), ("ldy", _I), ("top", _I), ("eps", _F)]


class GemmEpilogue(ctypes.Structure):
    _fields_ = [("resid32", _P), ("out2", _P), ("ldo2", _I), ("n_split", _I), ("scale", _F), ("glu_limit", _F),
                ("glu_alpha", _F), ("glu_bias", _F), ("softcap", _F), ("bias", _P)]


class TopkParams(ctypes.Structure):
    _fields_ = [("logits", _P), ("ws_val", _P), ("ws_idx", _P), ("out_val", _P), ("out_idx", _P),
                ("step_ptr", _P), ("status", _P), ("peer_buf", ctypes.c_uint64 * MAX_RANKS),
                ("timeout_ns", ctypes.c_ulonglong),
                ("M", _I), ("V", _I), ("ld", _I), ("k", _I), ("chunks", _I), ("chunk_size", _I),
                ("vocab_start", _I), ("tp", _I), ("rank", _I), ("order", _I), ("m_cap", _I)]


class ArRowsParams(ctypes.Structure):
    _fields_ = [("part_peer", ctypes.c_uint64 * MAX_RANKS), ("part_mc", ctypes.c_uint64),
                ("flag_peer", ctypes.c_uint64 * MAX_RANKS), ("resid", _P), ("h_out", _P), ("norm_w", _P), ("xh", _P),
                ("xl", _P), ("xscale", _P), ("xn", _P), ("step_ptr", _P), ("status", _P),
                ("timeout_ns", ctypes.c_ulonglong), ("M", _I), ("N", _I), ("tp", _I), ("rank", _I), ("order", _I),
                ("mode", _I), ("eps", _F), ("rows_cap", _I), ("two_shot", _I)]


class EditParams(ctypes.Structure):
    _fields_ = [("logits", _P), ("row_slot", _P), ("add_rows", _P), ("add_valid", _P), ("pen_ids", _P), ("pen_cnt", _P),
                ("pen_rp", _P), ("M", _I), ("V", _I), ("ld", _I), ("pen_cap", _I), ("chunk", _I)]


class SampleParams(ctypes.Structure):
    _fields_ = [("cand_val", _P), ("cand_idx", _P), ("temperature", _P), ("top_k", _P), ("top_p", _P), ("u", _P),
                ("out_tok", _P), ("status_src", _P), ("M", _I), ("n_cand", _I)]


_l.register("ti_ar_rows_params_size", _I, [], "hybrid")
_l.register("ti_ar_rows", _I, [ctypes.POINTER(ArRowsParams), _P], "hybrid")
_l.register("ti_edit_params_size", _I, [])
_l.register("ti_sample_params_size", _I, [])
_l.register("ti_logits_edit", _I, [ctypes.POINTER(EditParams), _P])
_l.register("ti_sample", _I, [ctypes.POINTER(SampleParams), _P])
_l.register("ti_embed", _I, [_P, _P, _P, _I, _I, _I, _P, _P])
_l.register("ti_rmsnorm", _I, [_P, _P, _P, _P, _P, _I, _I, _F, _I, _P])
_l.register("ti_act_mul", _I, [_P, _P, _P, _I, _I, _I, _I, _I, _I, _P])
_l.register("ti_swiglu_interleaved", _I, [_P, _P, _I, _I, _I, _I, _P])
_l.register("ti_gdn_params_size", _I, [], "hybrid")
_l.register("ti_gdn_step", _I, [ctypes.POINTER(GdnParams), _I, _I, _I, _I, _I, _P], "hybrid")
_l.register("ti_gdn_chunk_params_size", _I, [], "hybrid")
_l.register("ti_gdn_chunk_ws_bytes", _I, [_I, _I, _I], "hybrid")
_l.register("ti_gdn_chunked", _I, [ctypes.POINTER(GdnChunkParams), _I, _I, _I, _I, _I, _P], "hybrid")
_l.register("ti_qkv_prep_params_size", _I, [], "attention")
_l.register("ti_attn_params_size", _I, [], "attention")
_l.register("ti_qkv_prep", _I, [ctypes.POINTER(QkvPrepParams), _I, _I, _P], "attention")
_l.register("ti_attn_paged", _I, [ctypes.POINTER(AttnParams), _I, _I, _P], "attention")
_l.register("ti_attn_prefill", _I, [_P, _I, _P, _P, _I, _P, _P, _P, _P, _P, _I, _P, _P, _I, _I, _I, _I, _F, _I, _I, _F, _F,
                                _I, _P, _P, _I, _I, _I, _F, _I, _I, _P, _P], "attention")
_l.register("ti_rope_unit_params_size", _I, [], "attention")
_l.register("ti_rope_unit", _I, [ctypes.POINTER(RopeUnitParams), _I, _P], "attention")
_l.register("ti_attn_general_params_size", _I, [], "attention")
_l.register("ti_attn_general", _I, [ctypes.POINTER(AttnGeneralParams), _I, _P], "attention")
_l.register("ti_gla_params_size", _I, [], "gla")
_l.register("ti_gla_step", _I, [ctypes.POINTER(GlaParams), _I, _I, _I, _I, _P], "gla")
_l.register("ti_gla_chunk_size", _I, [_I], "gla")
_l.register("ti_gla_chunked", _I, [ctypes.POINTER(GlaParams), _I, _I, _P], "gla")
_l.register("ti_gla_finish", _I, [ctypes.POINTER(GlaParams), _I, _I, _I, _P], "gla")
_l.register("ti_norm_rope_params_size", _I, [], "attention")
_l.register("ti_norm_rope", _I, [ctypes.POINTER(NormRopeParams), _I, _P], "attention")
_l.register("ti_conv_params_size", _I, [], "conv")
_l.register("ti_conv", _I, [ctypes.POINTER(ConvParams), _I, _P], "conv")
_l.register("ti_ssd_params_size", _I, [], "ssd")
_l.register("ti_ssd_step", _I, [ctypes.POINTER(SsdParams), _I, _I, _I, _P], "ssd")
_l.register("ti_ssd_finish", _I, [ctypes.POINTER(SsdParams), _I, _I, _P], "ssd")
_l.register("ti_ssd_chunk_size", _I, [_I], "ssd")
_l.register("ti_ssd_chunked", _I, [ctypes.POINTER(SsdParams), _I, _P], "ssd")
_l.register("ti_delta_params_size", _I, [], "delta")
_l.register("ti_head_norm_params_size", _I, [], "delta")
_l.register("ti_delta_step", _I, [ctypes.POINTER(DeltaParams), _I, _I, _I, _I, _I, _P], "delta")
_l.register("ti_delta_chunk_size", _I, [_I], "delta")
_l.register("ti_delta_chunked", _I, [ctypes.POINTER(DeltaParams), _I, _I, _I, _P], "delta")
_l.register("ti_head_norm", _I, [ctypes.POINTER(HeadNormParams), _I, _I, _P], "delta")
_l.register("ti_gated_norm_params_size", _I, [], "rows")
_l.register("ti_gated_norm", _I, [ctypes.POINTER(GatedNormParams), _I, _I, _P], "rows")
_l.register("ti_moe_route_params_size", _I, [], "moe")
_l.register("ti_moe_route", _I, [ctypes.POINTER(MoeRouteParams), _P], "moe")
_l.register("ti_moe_norm_route", _I, [ctypes.POINTER(ResidNormParams), ctypes.POINTER(MoeRouteParams), _P, _P, _P, _I, _P], "moe")
_l.register("ti_moe_permute", _I, [_P, _I, _I, _P, _P, _P, _P, _P, _I, _I, _I, _I, _P], "moe")
_l.register("ti_gemm_grouped_bf16", _I, [_P, _I, _I, _I, _I, _P, _I, _P, _P, _I, _I, _P, _I, _I, _P, _P, _P], "moe")
_l.register("ti_gemm_grouped_w8a16", _I, [_P, _P, _I, _I, _I, _I, _P, _P, _P, _I, _P, _P, _I, _I, _P, _I, _I, _P, _P, _P], "moe")
_l.register("ti_resid_norm_params_size", _I, [], "rows")
_l.register("ti_resid_norm", _I, [ctypes.POINTER(ResidNormParams), _I, _I, _P], "rows")
_l.register("ti_topk_params_size", _I, [])
_l.register("ti_topk", _I, [ctypes.POINTER(TopkParams), _P])
_l.register("ti_topk_merge", _I, [ctypes.POINTER(TopkParams), _P])
_l.register("ti_symm_alloc", _I, [ctypes.POINTER(_P), ctypes.c_size_t])
_l.register("ti_symm_free", _I, [_P])
_l.register("ti_ipc_handle_size", _I, [])
_l.register("ti_ipc_get_handle", _I, [_P, _P])
_l.register("ti_ipc_open", _I, [_P, ctypes.POINTER(_P)])
_l.register("ti_ipc_close", _I, [_P])
_l.register("ti_memset_async", _I, [_P, _I, ctypes.c_size_t, _P])
_l.register("ti_wait_flag_probe", _I, [_P, ctypes.c_uint, ctypes.c_ulonglong, _P, _P, _P])

_l.register("ti_quant_rows", _I, [_P, _I, _P, _F, _I, _I, _P, _P, _P, _P])
_l.register("ti_gemm_epilogue_size", _I, [])
_l.register("ti_gemm_bf16", _I, [_P, _I, _I, _I, _P, _I, _P, _P, _I, _I, _P, _P, ctypes.c_size_t, _P, _I, _P, _P])
_l.register("ti_gemm_w8a16", _I, [_P, _P, _I, _I, _I, _P, _P, _P, _I, _P, _P, _I, _I, _P, _P, ctypes.c_size_t, _P, _I, _P, _P])
_l.register("ti_latent_attn_params_size", _I, [], "latent")
_l.register("ti_latent_attn_splits", _I, [_I, _I], "latent")
_l.register("ti_latent_attn", _I, [ctypes.POINTER(LatentAttnParams), _I, _P], "latent")
_l.register("ti_latent_prefill", _I, [_P, _I, _I, _P, _I, _I, _P, _I, _P, _P, _I, _I, _P, _I, _I, _I, _I, _I, _I, _F, _P, _P], "latent")
_l.register("ti_embed_pos", _I, [_P, _P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _F, _F, _P, _P, _I, _P], "rows")
_l.register("ti_rmsnorm_f32", _I, [_P, _P, _P, _I, _I, _I, _F, _I, _P], "rows")
_l.register("ti_latent_store", _I, [_P, _I, _I, _P, _P, _P, _LL, _I, _I, _I, _F, _I, _P], "latent")
_l.register("ti_latent_rope", _I, [_P, _I, _I, _I, _I, _I, _P, _P, _I, _P, _P, _P, _LL, _I, _I, _I, _F, _I, _P], "latent")
_l.register("ti_latent_gather", _I, [_P, _P, _LL, _P, _I, _I, _I, _P], "latent")
_l.register("ti_head_product", _I, [_P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _I, _P], "latent")
_l.register("ti_gemm_f32", _I, [_P, _P, _P, _P, _P, _I, _I, _I, _I, _I, _I, _I, _I, _F, _F, _F, _F, _P, _P, _I, _F, _P, _P], "rows")

_PARAM_SIZES = {"base": (("ti_topk_params_size", TopkParams), ("ti_edit_params_size", EditParams),
                         ("ti_sample_params_size", SampleParams), ("ti_gemm_epilogue_size", GemmEpilogue)),
                "latent": (("ti_latent_attn_params_size", LatentAttnParams),),
                "rows": (("ti_resid_norm_params_size", ResidNormParams), ("ti_gated_norm_params_size", GatedNormParams)),
                "attention": (("ti_qkv_prep_params_size", QkvPrepParams), ("ti_attn_params_size", AttnParams),
                              ("ti_rope_unit_params_size", RopeUnitParams), ("ti_attn_general_params_size", AttnGeneralParams),
                              ("ti_norm_rope_params_size", NormRopeParams)),
                "conv": (("ti_conv_params_size", ConvParams),),
                "ssd": (("ti_ssd_params_size", SsdParams),),
                "delta": (("ti_delta_params_size", DeltaParams), ("ti_head_norm_params_size", HeadNormParams)),
                "gla": (("ti_gla_params_size", GlaParams),),
                "moe": (("ti_moe_route_params_size", MoeRouteParams),),
                "hybrid": (("ti_gdn_params_size", GdnParams), ("ti_gdn_chunk_params_size", GdnChunkParams),
                           ("ti_ar_rows_params_size", ArRowsParams), ("ti_gemv_params_size", GemvParams),
                           ("ti_chain_params_size", ChainParams))}
_checked = set()


def L(*groups: str):
    """The kernel libraries; the named groups (default: what the hybrid family uses) are loaded now, with their parameter
    blocks checked against the Python structures."""
    lib = _l.lib()
    groups = groups or ("base", "attention", "hybrid")
    if not _checked.issuperset(groups):
        _l.build_groups(*groups)
        for g in groups:
            for fn, st in _PARAM_SIZES.get(g, ()):
                if getattr(lib, fn)() != ctypes.sizeof(st):
                    raise RuntimeError(f"{st.__name__} layout mismatch between Python and CUDA")
            _checked.add(g)
    return lib


# ------------------------------------------------------------------------------------ GEMV
class LinearW:
    """A weight matrix in kernel layout: 512-byte tiles [N/8][K/64 or K/32][8][64 B] (+ bf16 row scales)."""

    def __init__(self, w: torch.Tensor, quantize: bool, device="cuda"):
        from ..models.weights import pad_rows, quantize_int8_rowwise, tile_bf16, tile_int8
        self.N, self.K = w.shape
        w = pad_rows(w.to(device), 8)
        self.n_pad = w.shape[0]
        if quantize:
            assert self.K % 64 == 0, self.K
            q, s = quantize_int8_rowwise(w)
            self.tiles = tile_int8(q)
            self.scale = s.contiguous()
            self.wt, self.tile_k = W_INT8, 64
        else:
            assert self.K % 32 == 0, self.K
            self.tiles = tile_bf16(w.to(torch.bfloat16))
            self.scale = None
            self.wt, self.tile_k = W_BF16, 32
        self.KB = self.K // self.tile_k
        self.n_tiles = self.n_pad // 8

    def state(self) -> dict:
        """Everything needed to rebuild this object without the source weight (on-disk shard cache)."""
        return {"tiles": self.tiles, "scale": self.scale, "N": self.N, "K": self.K, "n_pad": self.n_pad, "wt": self.wt}

    @classmethod
    def from_state(cls, d: dict, device="cuda") -> "LinearW":
        w = cls.__new__(cls)
        w.N, w.K, w.n_pad, w.wt = d["N"], d["K"], d["n_pad"], d["wt"]
        w.tiles = d["tiles"].to(device)
        w.scale = None if d["scale"] is None else d["scale"].to(device)
        w.tile_k = 64 if w.wt == W_INT8 else 32
        w.KB = w.K // w.tile_k
        w.n_tiles = w.n_pad // 8
        return w

    def dense(self) -> torch.Tensor:
        """Row-major bf16 copy [N, K] (tests and the prefill GEMM baseline)."""
        from ..models.weights import untile_int8
        if self.wt == W_INT8:
            return (untile_int8(self.tiles).float() * self.scale.float()[:, None])[:self.N].to(torch.bfloat16)
        nt, kt = self.tiles.shape[:2]
        return self.tiles.permute(0, 2, 1, 3).reshape(nt * 8, kt * 32)[:self.N]

    def nbytes(self) -> int:
        return self.tiles.numel() * self.tiles.element_size()


def _limb_stride(kslice: int) -> int:
    return kslice + ((64 - (kslice % 128)) + 128) % 128


def x_smem_bytes(wt: int, xmode: int, M: int, K: int, kslice: int) -> int:
    """Shared memory the staged activations take (must mirror x_smem_bytes_impl in gemv_w8a16.cu)."""
    b = 0
    if wt == W_INT8:
        b = 2 * M * _limb_stride(kslice)
    elif xmode == XNORM:
        b = (16 if M > 8 else 8) * (K + 8) * 2
    return (b + 2048 + 127) // 128 * 128


PART_BYTES = 0
SMEM_LIMIT = 227 * 1024 - 4096      # dynamic shared memory of the GEMV kernel (4 KB of the 227 are static)
GEMV_TPS = int(os.environ.get("TI_GEMV_TPS", "8"))       # must match the -DTI_GEMV_TPS the library was built with
_RING_CHOICES = tuple((GEMV_TPS, s) for s in range(48 // GEMV_TPS, 0, -1))


def plan_gemv(wt: int, xmode: int, M: int, n_tiles: int, KB: int, ncta: int = NUM_SMS):
    """(R, tps, stages) or None when M rows of this K do not fit in shared memory.
    R: row tiles per unit; (tps, stages): geometry of the per-warp weight ring that fits beside the staged
    activations and the partial-sum buffers in 227 KB."""
    tk = 64 if wt == W_INT8 else 32
    xb = x_smem_bytes(wt, xmode, M, KB * tk, KB * tk)
    R = 2 if n_tiles >= 8 * ncta * GEMV_WARPS else 1
    for tps, stages in _RING_CHOICES:
        if xb + PART_BYTES + GEMV_WARPS * (stages * (tps * 512 + 8) + 64) <= SMEM_LIMIT:
            return R, tps, stages
    return None


TEAM_BYTES = 2 * GEMV_WARPS * 32 * 16      # exchange buffer of team mode (must mirror kTeamBytes)


def plan_team(n_tiles: int, KB: int, R: int, team: int | None = None, ncta: int = NUM_SMS) -> int:
    """Team size T for a product: how many adjacent warps of a CTA share one unit, each streaming a slice of k.
    A product with fewer units than warps would leave warps (and the bytes they keep in flight) idle.
    `team` (or TI_GEMV_T) forces a size.

    Cost model (in 512-byte tiles a warp streams one after the other): a CTA holds GEMV_WARPS // T whole teams,
    the units are dealt to the teams in waves, a unit costs ceil(KB / T) tiles per warp plus a fixed part (team
    exchange and epilogue, about six tiles' worth).  Measured on the 27B layer at one row (chain of the four layer
    products): out_proj / down with T = 2 -> 91.4 us, T = 3 -> 87.5 us, T = 5 or 16 -> 90-95 us; the half shards
    of a 2-way tensor-parallel group 60.7 -> 58.2 us."""
    if team is None and "TI_GEMV_T" in os.environ:
        team = int(os.environ["TI_GEMV_T"])
    U = -(-n_tiles // R)
    if team is not None:
        return team if KB >= team else 1
    W = ncta * GEMV_WARPS
    if U >= 0.8 * W:
        return 1
    fixed = 6
    best, best_cost = 1, -(-U // W) * (KB + fixed)
    for T in range(2, GEMV_WARPS + 1):
        if KB < 8 * T:                       # a slice shorter than one ring stage is all overhead
            break
        teams = (GEMV_WARPS // T) * ncta
        cost = -(-U // teams) * (-(-KB // T) + fixed)
        if cost < 0.97 * best_cost:          # near-ties go to the smaller team
            best, best_cost = T, cost
    return best


def max_rows(wt: int, xmode: int, K: int) -> int:
    """Largest row count (<= 16) one launch can take for this K."""
    tk = 64 if wt == W_INT8 else 32
    for m in (16, 12, 8, 6, 4, 3, 2, 1):
        if plan_gemv(wt, xmode, m, 1024, K // tk) is not None:
            return m
    raise ValueError(f"K={K} does not fit in shared memory even for one row")


_STATUS = None


def status_ptr() -> int:
    """A process-wide device word that kernels OR error bits into when no communicator supplies one."""
    global _STATUS
    if _STATUS is None:
        _STATUS = torch.zeros(4, dtype=torch.int32, device="cuda")
    return _STATUS.data_ptr()


class GemvWorkspace:
    """Split-k partial buffer and per-tile arrival counters shared by all GEMV launches of a stream."""

    def __init__(self, device="cuda", max_units: int = 1 << 16, max_tiles: int = 1 << 16):
        self.ws = torch.empty(max_units * 128, dtype=torch.float32, device=device)
        self.counters = torch.zeros(max_tiles, dtype=torch.int32, device=device)
        self.sched = torch.zeros(128, dtype=torch.int32, device=device)     # dynamic unit scheduling state
        self.max_units, self.max_tiles = max_units, max_tiles


_DEFAULT_WS = None


def default_workspace():
    global _DEFAULT_WS
    if _DEFAULT_WS is None:
        _DEFAULT_WS = GemvWorkspace()
    return _DEFAULT_WS


def make_gemv_params(W: LinearW, x, out, M, *, xmode=XGLOBAL, epi=EPI_STORE, norm_w=None, resid=None, ws=None,
                     eps=1e-6, ldx=None, ldo=None, comm=None, order=0, ncta=NUM_SMS, team=None, xll=False,
                     out_idx=None) -> GemvParams:
    p = GemvParams()
    p.w, p.scale, p.x, p.norm_w = ptr(W.tiles), ptr(W.scale), ptr(x), ptr(norm_w)
    p.out, p.resid, p.out_idx = ptr(out), ptr(resid), ptr(out_idx)
    plan = plan_gemv(W.wt, xmode, M, W.n_tiles, W.KB, ncta)
    if plan is None:
        raise ValueError(f"{M} rows of K={W.K} do not fit in shared memory; split the rows (max_rows)")
    R, tps, stages = plan
    if ws is None:
        ws = default_workspace()
    p.M, p.N, p.n_tiles, p.K, p.KB, p.S, p.kb_per_split = M, W.N, W.n_tiles, W.K, W.KB, 1, W.KB
    p.ws = ptr(ws.ws)
    p.ldx = ldx if ldx is not None else (x.stride(0) if x.dim() > 1 else W.K)
    p.ldo = ldo if ldo is not None else (out.stride(0) if out.dim() > 1 else W.N)
    p.eps = eps
    p.stages, p.T, p.tps, p.R = stages, plan_team(W.n_tiles, W.KB, R, team, ncta), tps, R
    p._xb = x_smem_bytes(W.wt, xmode, M, W.K, W.K)
    p.xmode, p.epi = xmode, epi
    p.xll = int(bool(xll))
    if ws is None:
        ws = default_workspace()
    p.sched = ptr(ws.sched)
    p.status = status_ptr()
    p.tp, p.rank, p.order, p.m_cap = 1, 0, order, 0
    if comm is not None and comm.tp > 1:
        p.tp, p.rank, p.m_cap = comm.tp, comm.rank, comm.m_cap
        for r in range(comm.tp):
            p.peer_ll[r] = comm.ll_ptrs[r]
        p.step_ptr, p.status, p.timeout_ns = comm.step_ptr, comm.status_ptr, comm.timeout_ns
    return p


def make_chain(params: list) -> ChainParams:
    """Up to MAX_CHAIN dependent products for one launch; the ring depth is the smallest of the ops'."""
    assert 1 <= len(params) <= MAX_CHAIN
    c = ChainParams()
    c.n_ops = len(params)
    # one ring geometry per launch: the one of the op that has the least room
    tps, stages = min((p.tps * p.stages, p.tps, p.stages) for p in params)[1:]
    # team mode needs its exchange buffer next to the rings: give up ring stages for it, or, failing that, teams
    xb = max(getattr(p, "_xb", 0) for p in params)
    while any(p.T > 1 for p in params) and xb + TEAM_BYTES + GEMV_WARPS * (stages * (tps * 512 + 8) + 64) > SMEM_LIMIT:
        if stages > 1:
            stages -= 1
        else:
            for p in params:
                p.T = 1
    for i, p in enumerate(params):
        p.tps, p.stages = tps, stages
        c.op[i] = p
    return c


def gemv_chain_launch(params: list, wt: int, ncta: int = NUM_SMS):
    c = make_chain(params)
    check(_l.lib().ti_gemv_chain(ctypes.byref(c), wt, ncta, stream()), "ti_gemv_chain")


def gemv_launch(p: GemvParams, wt: int, xmode: int = None, epi: int = None, ncta: int = NUM_SMS):
    if xmode is not None:
        p.xmode = xmode
    if epi is not None:
        p.epi = epi
    gemv_chain_launch([p], wt, ncta)


def gemv(W: LinearW, x: torch.Tensor, *, out=None, xmode=XGLOBAL, epi=EPI_STORE, norm_w=None, resid=None, ws=None,
         eps=1e-6, comm=None, order=0, team=None) -> torch.Tensor:
    """Convenience form (allocates `out`); loops over row chunks that fit in shared memory."""
    M = x.shape[0]
    step = max_rows(W.wt, xmode, W.K)
    if out is None:
        cols = W.N // 2 if epi == EPI_SWIGLU else W.N
        dt = torch.float32 if epi == EPI_F32 else torch.bfloat16
        out = torch.empty(M, cols, dtype=dt, device=x.device)
    for m0 in range(0, M, step):
        m = min(step, M - m0)
        p = make_gemv_params(W, x[m0:m0 + m], out[m0:m0 + m], m, xmode=xmode, epi=epi, norm_w=norm_w,
                             resid=None if resid is None else resid[m0:m0 + m], ws=ws, eps=eps,
                             ldx=x.stride(0), ldo=out.stride(0), comm=comm, order=order, team=team)
        gemv_launch(p, W.wt, xmode, epi)
    return out


# ------------------------------------------------------------------------------------ pointwise
def embed(ids, table, out, step_ptr=0):
    M, H = out.shape
    check(_l.lib().ti_embed(ptr(ids), ptr(table), ptr(out), M, H, table.shape[0], step_ptr, stream()), "ti_embed")


def rmsnorm(x, w, eps, *, add=None, out=None, r_out=None, one_plus=True):
    M, H = x.shape
    if out is None:
        out = torch.empty_like(x)
    check(_l.lib().ti_rmsnorm(ptr(x), ptr(add), ptr(w), ptr(out), ptr(r_out), M, H, eps, int(one_plus), stream()), "ti_rmsnorm")
    return out


def act_mul(a, b, out=None, mode=0):
    M, n = a.shape
    if out is None:
        out = torch.empty(M, n, dtype=torch.bfloat16, device=a.device)
    check(_l.lib().ti_act_mul(ptr(a), ptr(b), ptr(out), M, n, a.stride(0), b.stride(0), out.stride(0), mode, stream()), "ti_act_mul")
    return out


def swiglu_interleaved(gu, out=None):
    M, n2 = gu.shape
    if out is None:
        out = torch.empty(M, n2 // 2, dtype=torch.bfloat16, device=gu.device)
    check(_l.lib().ti_swiglu_interleaved(ptr(gu), ptr(out), M, n2 // 2, gu.stride(0), out.stride(0), stream()), "ti_swiglu")
    return out


# ------------------------------------------------------------------------------------ launches by params
def gdn_step(p: GdnParams, num_seqs: int, dk: int, dv: int, state_bf16: bool, split: bool = False, single: bool = False,
             staged: bool = False):
    """single: every sequence has exactly one token (decode): the single-pass kernels (one block per head and sequence;
    for large batches column-split blocks, or, with `staged` or when snapshots are wanted, blocks that walk several
    sequences with the state staged through shared memory).  split: the state columns of a head go to a cluster of
    blocks (prefill; optional)."""
    mode = (3 if staged else 2) if single else int(split)
    if not p.status:
        p.status = status_ptr()
    check(_l.lib().ti_gdn_step(ctypes.byref(p), num_seqs, dk, dv, int(state_bf16), mode, stream()), "ti_gdn_step")


GDN_CHUNK = 64


def gdn_chunk_table(cu_seqlens, snapshot_rel=None, snapshot_entry=None):
    """Chunk table of the chunked DeltaNet prefill: every sequence is cut into chunks of at most 64 tokens that
    also end wherever a state snapshot is wanted.  `snapshot_rel[s]`: token counts (relative to the start of the
    step) after which sequence s snapshots, `snapshot_entry[s]`: the entries of the snapshot buffers.
    Returns int32 tensors (ck [4, nc] = sequence | first flat token | tokens | snapshot entry or -1, seq_ck [S+1])."""
    seq, tok0, ntok, snap, seq_ck = [], [], [], [], [0]
    for s in range(len(cu_seqlens) - 1):
        t0, t1 = cu_seqlens[s], cu_seqlens[s + 1]
        pts = {}
        if snapshot_rel is not None:
            for r, e in zip(snapshot_rel[s], snapshot_entry[s]):
                if 0 < r <= t1 - t0:
                    pts[r] = e
        cuts = sorted(set(range(GDN_CHUNK, t1 - t0, GDN_CHUNK)) | set(pts) | {t1 - t0})
        # chunks never straddle a snapshot point; between two cuts they are at most 64 tokens long
        a = 0
        for c in cuts:
            while a < c:
                n = min(GDN_CHUNK, c - a)
                seq.append(s); tok0.append(t0 + a); ntok.append(n)
                a += n
                snap.append(pts.get(a, -1))
        seq_ck.append(len(seq))
    return torch.tensor([seq, tok0, ntok, snap], dtype=torch.int32), torch.tensor(seq_ck, dtype=torch.int32)


class GdnChunkWorkspace:
    """Fragment-order operands of the scan kernel for up to `nc * hv` (chunk, head) pairs; grows on demand."""

    def __init__(self, device):
        self.device, self.cap, self.bufs = device, 0, None

    def get(self, n_items: int, dk: int, dv: int):
        if n_items > self.cap or self.bufs is None or self.key != (dk, dv):
            lib = _l.lib()
            sizes = [lib.ti_gdn_chunk_ws_bytes(dk, dv, i) for i in range(6)]
            cap = max(n_items, 2 * self.cap)
            self.bufs = [torch.empty(cap * sz, dtype=torch.uint8, device=self.device) for sz in sizes]
            self.cap, self.key = cap, (dk, dv)
        return self.bufs


def gdn_chunked(p: GdnChunkParams, num_seqs: int, T: int, dk: int, dv: int, state_bf16: bool):
    check(_l.lib().ti_gdn_chunked(ctypes.byref(p), num_seqs, T, dk, dv, int(state_bf16), stream()), "ti_gdn_chunked")


def qkv_prep(p: QkvPrepParams, T: int, D: int):
    if not p.status:
        p.status = status_ptr()
    check(_l.lib().ti_qkv_prep(ctypes.byref(p), T, D, stream()), "ti_qkv_prep")


def attn_paged(p: AttnParams, D: int, DV: int = None):
    """D, DV: sizes of a query / key head and of a value head (64, 128 or 256)."""
    if not p.status:
        p.status = status_ptr()
    check(_l.lib().ti_attn_paged(ctypes.byref(p), D, D if DV is None else DV, stream()), "ti_attn_paged")


def attn_prefill(q, kcache, vcache, num_blocks, block_tables, positions, tiles, gate_src, out, *, hq, hkv, D,
                 max_blocks, ld, DV=None, scale=None, softcap=0.0, qk_max=0.0, window=0, slopes=None, head_gate=None, gcol=0, out_scale=1.0,
                 gate_col=0, gate_stride=0):
    """Causal GQA attention of prefill query tiles on the tcgen05 tensor cores (ops/csrc/attn_prefill.cu).
    `tiles`: int32 [3, n] = (sequence, first flat token, tokens <= 128) per tile, longest KV first.  DV: size of a value
    head (default D); softcap: scores become softcap * tanh(scale q.k / softcap); qk_max: a bound of |q.k| where there is
    one (it selects a cheaper softmax); gate_src None: no output gate, else rows of pitch `ld` with the gates of head h at column
    gate_col + h * gate_stride (stride 0: h * 2 D + D).  window: keys seen (0: all); slopes: fp32 [hq], taken
    off a score per token of distance; head_gate: rows whose column gcol + h gates head h; out_scale: factor of the output."""
    n = tiles.shape[1]
    scale = D ** -0.5 if scale is None else scale
    check(_l.lib().ti_attn_prefill(ptr(q), q.shape[0], ptr(kcache), ptr(vcache), num_blocks, ptr(block_tables), ptr(positions),
                              ptr(tiles[0]), ptr(tiles[1]), ptr(tiles[2]), n, ptr(gate_src), ptr(out), hq, hkv,
                              max_blocks, ld, scale, D, D if DV is None else DV, softcap, qk_max, window, ptr(slopes), ptr(head_gate),
                              0 if head_gate is None else head_gate.stride(0), gcol, out.stride(0) if out.dim() == 2 else 0, out_scale, gate_col, gate_stride,
                              status_ptr(), stream()),
          "ti_attn_prefill")


AR_NONE, AR_LIMBS, AR_BF16 = 0, 1, 2


def ar_rows(comm, parity: int, M: int, N: int, resid, h_out, *, order: int, mode: int = AR_NONE, norm_w=None,
            limbs: "Limbs" = None, xn=None, eps: float = 1e-6, two_shot: int = 0):
    """All-reduce of the row-parallel partials in `comm`'s symmetric buffer `parity` + residual -> h_out, fused with
    the RMSNorm / activation-quantisation prologue of the consuming product (ops/csrc/fused_ar.cu).
    two_shot = 1: every rank first reduces its 1/tp of the rows and broadcasts the sums into all ranks' buffers, the
    row kernel then reads local memory (many rows on >= 4 ranks); 2 / 3 run only the first / second launch (tests
    that emulate the ranks one after the other on one GPU)."""
    p = ArRowsParams()
    for r in range(comm.tp):
        p.part_peer[r] = comm.part_ptrs[parity][r]
        p.flag_peer[r] = comm.flag_ptrs[r]
    p.part_mc = comm.part_mc[parity]
    p.resid, p.h_out, p.norm_w = ptr(resid), ptr(h_out), ptr(norm_w)
    if mode == AR_LIMBS:
        p.xh, p.xl, p.xscale = ptr(limbs.hi), ptr(limbs.lo), ptr(limbs.scale)
    elif mode == AR_BF16:
        p.xn = ptr(xn)
    p.step_ptr, p.status, p.timeout_ns = comm.step_ptr, comm.status_ptr, comm.timeout_ns
    p.M, p.N, p.tp, p.rank, p.order, p.mode, p.eps = M, N, comm.tp, comm.rank, order, mode, eps
    p.rows_cap = int(getattr(comm, "ar_rows", 0) or 0)
    p.two_shot = int(two_shot)
    check(_l.lib().ti_ar_rows(ctypes.byref(p), stream()), "ti_ar_rows")


def logits_edit(p: EditParams):
    check(_l.lib().ti_logits_edit(ctypes.byref(p), stream()), "ti_logits_edit")


def sample(p: SampleParams):
    check(_l.lib().ti_sample(ctypes.byref(p), stream()), "ti_sample")


def topk(p: TopkParams):
    check(_l.lib().ti_topk(ctypes.byref(p), stream()), "ti_topk")


def topk_merge(p: TopkParams):
    """Second stage only: merges the per-chunk candidates already in ws_val / ws_idx (written, for instance, by the
    arg-max epilogue of the lm_head GEMV: one candidate per row and CTA) and exchanges the winners between ranks."""
    check(_l.lib().ti_topk_merge(ctypes.byref(p), stream()), "ti_topk_merge")


# ------------------------------------------------------------------------------------ prefill GEMM (tcgen05)
GEPI_STORE, GEPI_SWIGLU, GEPI_ROWPAR, GEPI_F32, GEPI_RESID32, GEPI_SPLIT_GLU, GEPI_SPLIT_RELU2 = 0, 1, 2, 3, 4, 5, 6


def gemm_epilogue(*, resid32=None, out2=None, n_split=0, scale=1.0, glu=(math.inf, 1.0, 0.0), softcap=0.0, bias=None) -> GemmEpilogue:
    """Operands of the extended epilogues: an fp32 residual (GEPI_RESID32), the second output and the constants
    (limit, alpha, bias) of the clamped gated unit (GEPI_SPLIT_GLU; GEPI_SPLIT_RELU2 squares the positive part instead), a factor and a cap of the stored fp32 values (GEPI_F32), and an fp32 vector [N]
    added to the product first (any of them)."""
    return GemmEpilogue(ptr(resid32), ptr(out2), 0 if out2 is None else out2.stride(0), n_split, scale, *glu, softcap, ptr(bias))


class Limbs:
    """Activation rows split into two int8 planes plus the per-row value of one fixed-point unit."""

    def __init__(self, M: int, K: int, device):
        self.M, self.K = M, K
        self.hi = torch.empty(M, K, dtype=torch.int8, device=device)
        self.lo = torch.empty(M, K, dtype=torch.uint8, device=device)
        self.scale = torch.empty(M, dtype=torch.float32, device=device)


def _ref(struct):
    return None if struct is None else ctypes.addressof(struct)


def quant_rows(x: torch.Tensor, norm_w=None, eps: float = 1e-6, out: Limbs = None) -> Limbs:
    """Limb planes of x [M, K] (bf16, row stride x.stride(0)); RMSNorm(1+w) fused when norm_w is given."""
    M, K = x.shape
    if out is None:
        out = Limbs(M, K, x.device)
    check(_l.lib().ti_quant_rows(ptr(x), x.stride(0), ptr(norm_w), eps, M, K, ptr(out.hi), ptr(out.lo), ptr(out.scale),
                            stream()), "ti_quant_rows")
    return out


def gemm_w8a16(W: "LinearW", limbs: Limbs, *, out=None, epi=GEPI_STORE, resid=None, ex=None) -> torch.Tensor:
    """y = x W^T on the tcgen05 tensor cores for int8-tiled W and the limb planes of x (any M)."""
    assert W.wt == W_INT8 and limbs.K == W.K
    M = limbs.M
    if out is None:
        out = torch.empty(M, W.N // 2 if epi == GEPI_SWIGLU else W.N, dtype=torch.bfloat16, device=limbs.hi.device)
    part, count = _gemm_workspace(limbs.hi.device)
    check(_l.lib().ti_gemm_w8a16(ptr(W.tiles), ptr(W.scale), W.n_tiles, W.N, W.K, ptr(limbs.hi), ptr(limbs.lo),
                            ptr(limbs.scale), M, ptr(resid), ptr(out), out.stride(0), epi, status_ptr(), ptr(part),
                            part.numel() * 4, ptr(count), count.numel(), _ref(ex), stream()), "ti_gemm_w8a16")
    return out


def gemm_bf16(W: "LinearW", x: torch.Tensor, *, out=None, epi=GEPI_STORE, resid=None, ex=None) -> torch.Tensor:
    """y = x W^T on the tcgen05 tensor cores (kind::f16) for bf16-tiled W and bf16 x [M, K] with contiguous rows.
    epi GEPI_F32 stores fp32 (logits)."""
    assert W.wt == W_BF16 and x.shape[1] == W.K and x.stride(1) == 1 and x.stride(0) == W.K and x.dtype == torch.bfloat16
    M = x.shape[0]
    if out is None:
        cols = W.N // 2 if epi == GEPI_SWIGLU else W.N
        out = torch.empty(M, cols, dtype=torch.float32 if epi == GEPI_F32 else torch.bfloat16, device=x.device)
    part, count = _gemm_workspace(x.device)
    check(_l.lib().ti_gemm_bf16(ptr(W.tiles), W.n_tiles, W.N, W.K, ptr(x), M, ptr(resid), ptr(out), out.stride(0), epi,
                           status_ptr(), ptr(part), part.numel() * 4, ptr(count), count.numel(), _ref(ex), stream()), "ti_gemm_bf16")
    return out


_GEMM_WS = {}


def _gemm_workspace(device):
    """Split-k partials (fp32, 32 MB: 16 slices of 128 rows x 4096 columns, or fewer of wider products) and the
    per-tile arrival counters, one set per device; launches on one stream use them one after the other."""
    key = str(device)
    if key not in _GEMM_WS:
        _GEMM_WS[key] = (torch.empty(8 << 20, dtype=torch.float32, device=device),
                         torch.zeros(256, dtype=torch.int32, device=device))
    return _GEMM_WS[key]


# ------------------------------------------------------------------------------------ latent attention, fp32 residual
def _f32(t) -> int:
    assert t.dtype in (torch.float32, torch.bfloat16), t.dtype
    return int(t.dtype == torch.float32)


def embed_pos(ids, positions, embed, pos, norm_w, x, W, eps, step_ptr=0, scale=1.0, h=None):
    """x[m] (fp32) = rmsnorm(embed[ids[m]] + pos[positions[m]]) * norm_w * scale; `pos` and `norm_w` (no norm) may be None.  h: the
    row once more, in the activations' type."""
    check(_l.lib().ti_embed_pos(ptr(ids), ptr(positions), ptr(embed), ptr(pos), ptr(norm_w), ptr(x), x.shape[0], W, x.stride(0),
                                embed.shape[0], 0 if pos is None else pos.shape[0], eps, scale, step_ptr, ptr(h), _f32(embed), stream()), "ti_embed_pos")


def rmsnorm_f32(x, norm_w, y, W, eps):
    """y = rmsnorm(x) * norm_w for fp32 rows x [M, pitch] of true width W; y bf16 or fp32 of the same pitch."""
    assert x.stride(0) == y.stride(0) and norm_w.numel() == x.stride(0)
    check(_l.lib().ti_rmsnorm_f32(ptr(x), ptr(norm_w), ptr(y), x.shape[0], W, x.stride(0), eps, _f32(y), stream()), "ti_rmsnorm_f32")


def latent_rope(proj, H, dp, dim, col0, norm_w, inv_freq, positions, slots, cache, R, eps):
    """Turns dimensions dim .. dim + 2 * inv_freq.numel() of the H query heads (proj columns h * dp, in place), and stores
    [normalised latent of R columns | turned key part] of proj[:, col0:] in the slots of `cache` [blocks, 16, Rp]."""
    Rp = cache.shape[-1]
    assert norm_w.numel() >= R and cache.dtype == proj.dtype
    check(_l.lib().ti_latent_rope(ptr(proj), proj.stride(0), H, dp, dim, col0, ptr(norm_w), ptr(inv_freq), inv_freq.numel(), ptr(positions),
                                  ptr(slots), ptr(cache), cache.numel() // Rp, proj.shape[0], R, Rp, eps, _f32(proj), stream()),
          "ti_latent_rope")


def latent_store(proj, col0, norm_w, slots, cache, R, eps):
    """Normalised latents proj[:, col0 : col0 + R] into their slots of `cache` [blocks, 16, Rp]."""
    Rp = cache.shape[-1]
    assert norm_w.numel() == Rp and cache.dtype == proj.dtype
    check(_l.lib().ti_latent_store(ptr(proj), proj.stride(0), col0, ptr(norm_w), ptr(slots), ptr(cache), cache.numel() // Rp,
                                   proj.shape[0], R, Rp, eps, _f32(proj), stream()), "ti_latent_store")


def latent_gather(cache, slots, out):
    """Rows of the listed slots (int64) of `cache` [blocks, 16, Rp] -> out [n, Rp]."""
    Rp = cache.shape[-1]
    check(_l.lib().ti_latent_gather(ptr(cache), ptr(slots), cache.numel() // Rp, ptr(out), slots.numel(), Rp, _f32(cache), stream()),
          "ti_latent_gather")


def head_product(x, w, out, gate=None, gcol=0):
    """out[t, h] = w[h] x[t, h] per head (w [H, N, K]), times sigmoid(gate[t, gcol + h]) when a gate is given.  x and out
    are row views whose heads lie side by side."""
    H, N, K = w.shape
    check(_l.lib().ti_head_product(ptr(x), ptr(w), ptr(gate), ptr(out), x.shape[0], H, N, K, x.stride(0), out.stride(0),
                                   0 if gate is None else gate.stride(0), gcol, _f32(w), stream()), "ti_head_product")


def latent_rows(H: int) -> int:
    """Heads a block of the split latent attention takes."""
    return 32 if H > 16 else 16


def latent_nsplit(num_qg: int, H: int, Rp: int, window: int) -> int:
    """Splits of the key range (bf16, Rp <= 512): fill the SMs once, at least a tile of 64 keys each."""
    groups = -(-H // latent_rows(H))
    tiles = (window + 14) // 64 + 1 if window else 1 << 20
    return max(1, min(32, NUM_SMS // max(1, num_qg * groups), tiles))


def latent_part_floats(num_qg: int, H: int, Rp: int, nsplit: int) -> int:
    """Size of the partial-output buffer; the (max, sum) buffer has two floats per row of Rp."""
    return num_qg * -(-H // latent_rows(H)) * nsplit * latent_rows(H) * Rp


def latent_attn_splits(Rp: int, Ro: int) -> bool:
    """Whether a kernel with splits takes cache rows of Rp columns of which the first Ro are values (bf16)."""
    return bool(_l.lib().ti_latent_attn_splits(Rp, Ro))


def latent_attn(p: LatentAttnParams, f32: bool):
    """p.Ro 0: every column of a cache row is key and value."""
    if not p.status:
        p.status = status_ptr()
    p.Ro = p.Ro or p.Rp
    check(_l.lib().ti_latent_attn(ctypes.byref(p), int(f32), stream()), "ti_latent_attn")


def latent_prefill(q, kv, tiles, out, *, H, dp, vp, window, scale, sink=None, gate=None, gcol=0, status=0):
    """Windowed attention of prefill query tiles over expanded rows kv [Nk, H * dp keys | H * vp values] (bf16).
    `tiles`: int32 [5, n] = first flat token, tokens, its position, a row of kv, the position that row holds."""
    check(_l.lib().ti_latent_prefill(ptr(q), q.shape[0], q.stride(0), ptr(kv), kv.shape[0], kv.stride(0), ptr(tiles), tiles.shape[1],
                                     ptr(sink), ptr(gate), 0 if gate is None else gate.stride(0), gcol, ptr(out), out.stride(0),
                                     H, dp, vp, H * dp, window, scale, status or status_ptr(), stream()), "ti_latent_prefill")


def gemm_f32(w, x, *, out, epi=GEPI_F32, ex=None, groups=None):
    """y = x W^T in fp32 FMAs (w [N, K] row-major) with the GEPI_F32 / GEPI_RESID32 / GEPI_SPLIT_GLU / GEPI_SPLIT_RELU2 epilogues.  With
    `groups` w is [E, N, K] and the rows of x meet the matrices of the token tiles (of at most 64 rows)."""
    e = ex if ex is not None else gemm_epilogue()
    N, K = w.shape[-2:]
    check(_l.lib().ti_gemm_f32(ptr(w), ptr(x), e.resid32, ptr(out), e.out2, x.shape[0], N, K, x.stride(0), 0 if out is None else out.stride(0), e.ldo2,
                               e.n_split, epi, e.scale, e.glu_limit, e.glu_alpha, e.glu_bias,
                               *((0, 0, 0) if groups is None else (ptr(groups.tiles), ptr(groups.num_tiles), groups.tiles.shape[1])),
                               e.softcap, e.bias, stream()), "ti_gemm_f32")


def gated_norm(y, gate, x, w_out, h, W, eps, y2=None, w_y=None, w_y2=None, scale=1.0):
    """x += rmsnorm(sigmoid(gate) * Y) * w_out (fp32 rows) and h = x, with Y = y, or scale * (rmsnorm(y) * w_y + rmsnorm(y2) * w_y2)."""
    p = GatedNormParams()
    p.y, p.y2, p.gate, p.w_y, p.w_y2, p.w_out, p.x, p.h = (ptr(t) for t in (y, y2, gate, w_y, w_y2, w_out, x, h))
    p.W, p.P, p.ldy, p.ldg, p.eps, p.scale = W, x.stride(0), y.stride(0), gate.stride(0), eps, scale
    check(_l.lib().ti_gated_norm(ctypes.byref(p), x.shape[0], _f32(y), stream()), "ti_gated_norm")


def resid_norm(y, x, w_out, h, w_next, W, eps, routed=None):
    """x += rmsnorm(y) * w_out (fp32 rows; w_out None: x += y), then h = rmsnorm(x) * w_next unless w_next is None.  With `routed` (a
    TokenGroups after `moe_permute`) y holds the experts' rows and h the input of the identity experts."""
    p = _resid_params(y, x, w_out, h, w_next, W, eps, routed)
    check(_l.lib().ti_resid_norm(ctypes.byref(p), x.shape[0], _f32(h), stream()), "ti_resid_norm")


def _resid_params(y, x, w_out, h, w_next, W, eps, routed=None) -> ResidNormParams:
    p = ResidNormParams()
    p.y, p.x, p.w_out, p.w_next, p.h = ptr(y), ptr(x), ptr(w_out), ptr(w_next), ptr(h)
    if routed is not None:
        p.slot, p.weight, p.h_in, p.top = ptr(routed.slot), ptr(routed.weight), ptr(h), routed.top
    p.W, p.P, p.ldy, p.eps = W, x.stride(0), 0 if y is None else y.stride(0), eps
    return p


# ------------------------------------------------------------------------------------ rotated unit heads, plain attention
def rope_unit(p: RopeUnitParams, f32: bool):
    if not p.status:
        p.status = status_ptr()
    check(_l.lib().ti_rope_unit(ctypes.byref(p), int(f32), stream()), "ti_rope_unit")


def norm_rope(p: NormRopeParams, f32: bool):
    """Queries and keys normed over all their heads together, turned in neighbouring pairs; keys and values into the cache."""
    check(_l.lib().ti_norm_rope(ctypes.byref(p), int(f32), stream()), "ti_norm_rope")


def attn_general(p: AttnGeneralParams, f32: bool):
    if not p.status:
        p.status = status_ptr()
    check(_l.lib().ti_attn_general(ctypes.byref(p), int(f32), stream()), "ti_attn_general")


# ------------------------------------------------------------------------------------ gated linear attention
GLA_KEY_SIZES = (64, 128, 256, 512)     # key sizes the kernels are built for


def gla_step(p: GlaParams, num_seqs: int, dk: int, dv: int, f32: bool):
    check(_l.lib().ti_gla_step(ctypes.byref(p), num_seqs, dk, dv, int(f32), stream()), "ti_gla_step")


def gla_chunk_size(dk: int) -> int:
    """Tokens of a chunk for this key size (0: no chunked form)."""
    return _l.lib().ti_gla_chunk_size(dk)


def gla_chunk_table(cu_seqlens, seqs, chunk: int, snapshot_points=None):
    """Chunks of the listed sequences: every one is cut after `chunk` tokens, and where a state snapshot is wanted
    (`snapshot_points[s]`: {tokens into the step: entry of the snapshot buffers}).  Returns int32 tensors (ck [4, nc] =
    sequence | first flat token | tokens | snapshot entry or -1, rng [num_long + 1] = chunk range of every listed sequence)."""
    rows, rng = [], [0]
    for s in seqs:
        t0, n = cu_seqlens[s], cu_seqlens[s + 1] - cu_seqlens[s]
        pts = snapshot_points[s] if snapshot_points else {}
        a = 0
        while a < n:
            b = min([a + chunk, n] + [x for x in pts if a < x])
            rows.append((s, t0 + a, b - a, pts.get(b, -1)))
            a = b
        rng.append(len(rows))
    return torch.tensor(rows, dtype=torch.int32).t().contiguous(), torch.tensor(rng, dtype=torch.int32)


class GlaWorkspace:
    """Running decays and chunk states of the chunked form; grows on demand."""

    def __init__(self, device):
        self.device, self.g, self.s = device, None, None

    def get(self, nc: int, H: int, dk: int, dv: int):
        ng, ns = nc * H * gla_chunk_size(dk) * dk, nc * H * dk * dv
        if self.g is None or self.g.numel() < ng:
            self.g = torch.empty(ng, dtype=torch.float32, device=self.device)
        if self.s is None or self.s.numel() < ns:
            self.s = torch.empty(ns, dtype=torch.float32, device=self.device)
        return self.g, self.s


def gla_chunked(p: GlaParams, dk: int, dv: int):
    """Outputs and states of the sequences with chunks (bf16 projections); three kernels."""
    check(_l.lib().ti_gla_chunked(ctypes.byref(p), dk, dv, stream()), "ti_gla_chunked")


def gla_finish(p: GlaParams, T: int, dv: int, f32: bool):
    check(_l.lib().ti_gla_finish(ctypes.byref(p), T, dv, int(f32), stream()), "ti_gla_finish")


# ------------------------------------------------------------------------------------ short convolutions
CONV_TILE = 16          # tokens of a tile of the convolution (kConvTile in conv.cu)


def conv_tiles(cu_seqlens) -> torch.Tensor:
    """int32 [3, n] = sequence | first flat token | tokens: the sequences of a step cut into tiles."""
    rows = [(s, a, min(CONV_TILE, t1 - a)) for s, (t0, t1) in enumerate(zip(cu_seqlens[:-1], cu_seqlens[1:])) for a in range(t0, t1, CONV_TILE)]
    return torch.tensor(rows, dtype=torch.int32).view(-1, 3).t().contiguous()


def conv(p: ConvParams, f32: bool):
    """Causal convolution of a step's tokens (two kernels when p.cu is set, else one)."""
    check(_l.lib().ti_conv(ctypes.byref(p), int(f32), stream()), "ti_conv")


# ------------------------------------------------------------------------------------ delta rules
def delta_chunk_size(dk: int) -> int:
    """Tokens of a chunk for this key size (0: no chunked form)."""
    return _l.lib().ti_delta_chunk_size(dk)


class DeltaWorkspace:
    """The matrices of the chunks (ops/csrc/delta_chunk.cu); grows on demand."""

    def __init__(self, device):
        self.device, self.w = device, [None] * 4

    def get(self, nc: int, H: int, dk: int, dv: int):
        sizes = (nc * H * dk * dk, nc * H * delta_chunk_size(dk) * dk, nc * H * dk * dv, nc * H * dk)
        for i, n in enumerate(sizes):
            if self.w[i] is None or self.w[i].numel() < n:
                self.w[i] = torch.empty(n, dtype=torch.float32, device=self.device)
        return self.w


def delta_step(p: DeltaParams, num_seqs: int, dk: int, dv: int, general: bool, f32: bool):
    check(_l.lib().ti_delta_step(ctypes.byref(p), num_seqs, dk, dv, int(general), int(f32), stream()), "ti_delta_step")


def delta_chunked(p: DeltaParams, dk: int, dv: int, general: bool):
    """Outputs and states of the sequences with chunks (bf16 inputs); three kernels."""
    check(_l.lib().ti_delta_chunked(ctypes.byref(p), dk, dv, int(general), stream()), "ti_delta_chunked")


def head_norm(o, gate, g_col, norm, out, vdim, eps, silu: bool):
    """out[t, h] = rmsnorm(o[t, h]) * norm * (silu or sigmoid)(gate): o [T, H, dv] fp32, gate rows with the heads at column g_col,
    norm [dv] or [H, dv], out rows with head h at column h * dv."""
    p = HeadNormParams()
    p.o, p.gate, p.norm, p.out = ptr(o), ptr(gate), ptr(norm), ptr(out)
    p.ld, p.ldo, p.g_col, p.H, p.dv = gate.stride(0), out.stride(0), g_col, o.shape[1], o.shape[2]
    p.vdim, p.norm_stride, p.silu, p.eps = vdim, 0 if norm.dim() == 1 else o.shape[2], int(silu), eps
    check(_l.lib().ti_head_norm(ctypes.byref(p), o.shape[0], _f32(gate), stream()), "ti_head_norm")


# ------------------------------------------------------------------------------------ state-space mixer
SSD_STATE_SIZES = (64, 128, 256, 512)     # state sizes the kernels are built for


def ssd_chunk_size(Np: int) -> int:
    """Tokens of a chunk for this state size (0: no chunked form)."""
    return _l.lib().ti_ssd_chunk_size(Np)


class SsdWorkspace:
    """Running decays, step sizes and chunk states of the chunked form; grows on demand."""

    def __init__(self, device):
        self.device, self.g, self.s = device, None, None

    def get(self, nc: int, H: int, Np: int, vp: int):
        ng, ns = nc * H * 2 * ssd_chunk_size(Np), nc * H * Np * vp
        if self.g is None or self.g.numel() < ng:
            self.g = torch.empty(ng, dtype=torch.float32, device=self.device)
        if self.s is None or self.s.numel() < ns:
            self.s = torch.empty(ns, dtype=torch.float32, device=self.device)
        return self.g, self.s


def ssd_step(p: SsdParams, num_seqs: int, Np: int, f32: bool):
    check(_l.lib().ti_ssd_step(ctypes.byref(p), num_seqs, Np, int(f32), stream()), "ti_ssd_step")


def ssd_chunked(p: SsdParams, Np: int):
    """Outputs and states of the sequences with chunks (bf16 inputs); three kernels."""
    check(_l.lib().ti_ssd_chunked(ctypes.byref(p), Np, stream()), "ti_ssd_chunked")


def ssd_finish(p: SsdParams, T: int, f32: bool):
    """silu(z) gate and the norm of equal parts."""
    check(_l.lib().ti_ssd_finish(ctypes.byref(p), T, int(f32), stream()), "ti_ssd_finish")


# ------------------------------------------------------------------------------------ experts
class TokenGroups:
    """Routing of up to T tokens to `top` of E experts: chosen experts, weights, rows, and the table of token tiles the
    grouped products run on.  `counters` (see `moe_counters`) may be shared by everything on one stream."""

    def __init__(self, T: int, E: int, choices: int, top: int, counters, f32: bool, device, fixed: bool = False):
        """`fixed`: every expert has T rows of its own (for `moe_norm_route`), else the experts' rows follow each other."""
        self.T, self.E, self.choices, self.top, self.counters = T, E, choices, top, counters
        self.row_stride, self.rows = T if fixed else 0, E * T if fixed else T * top
        mean = T * top / choices                           # rows of an expert
        self.tile = 64 if f32 else 32 if mean <= 24 else 64 if mean <= 96 else 128
        n = T * top // self.tile + min(E, T * top)
        self.buf = torch.zeros(4, T * top, dtype=torch.int32, device=device)
        self.ids, self.pos, self.slot = self.buf[0], self.buf[1], self.buf[2]
        self.weight = self.buf[3].view(torch.float32)
        self.tiles = torch.zeros(3, n, dtype=torch.int32, device=device)
        self.num_tiles = torch.zeros(1, dtype=torch.int32, device=device)
        self.first = torch.zeros(E, dtype=torch.int32, device=device)


def moe_counters(max_experts: int, device):
    """Arrival counters of the routing kernel, zero between launches."""
    return torch.zeros(max_experts + 1, dtype=torch.int32, device=device)


def moe_route(g: TokenGroups, logits, correction, groups: int, keep: int, valid=None):
    """Chooses the experts of every row of `logits` [T, >= choices] (fp32) and lays out the token tiles.  correction None:
    no corrections, and the weights are a softmax over the chosen logits alone."""
    p = _route_params(g, correction, groups, keep, valid)
    p.logits, p.ldl = ptr(logits), logits.stride(0)
    check(_l.lib().ti_moe_route(ctypes.byref(p), stream()), "ti_moe_route")


NORM_ROUTE_MAX_WIDTH = 8192      # columns of a row that `moe_norm_route` takes


def moe_norm_route(y, x, w_out, h, w_next, W, eps, g: TokenGroups, router, correction, groups: int, keep: int, xs, valid=None):
    """`resid_norm` and, for the rows h it makes, the router product, `moe_route` and `moe_permute` (into xs) in one kernel,
    for few tokens and fixed rows (y None: x is complete, nothing is added).  router: [choices, P] in the type of h."""
    r, p = _resid_params(y, x, w_out, h, w_next, W, eps), _route_params(g, correction, groups, keep, valid)
    assert router.shape == (g.choices, x.stride(0)) and router.dtype == h.dtype and xs.shape[0] == g.rows and g.row_stride == g.T
    check(_l.lib().ti_moe_norm_route(ctypes.byref(r), ctypes.byref(p), ptr(router), ptr(g.slot), ptr(xs), _f32(h), stream()), "ti_moe_norm_route")


def _route_params(g: TokenGroups, correction, groups: int, keep: int, valid) -> MoeRouteParams:
    p = MoeRouteParams()
    p.correction, p.valid, p.ids, p.weight, p.pos = ptr(correction), ptr(valid), ptr(g.ids), ptr(g.weight), ptr(g.pos)
    p.counts, p.ticket, p.first, p.tiles, p.num_tiles = ptr(g.counters) + 4, ptr(g.counters), ptr(g.first), ptr(g.tiles), ptr(g.num_tiles)
    p.M, p.E, p.identity, p.top, p.groups, p.keep = g.T, g.E, g.choices - g.E, g.top, groups, keep
    p.tile_rows, p.max_tiles, p.row_stride = g.tile, g.tiles.shape[1], g.row_stride
    return p


def moe_permute(g: TokenGroups, h, xs):
    """Rows of h [T, P] to their places in xs [T * top, P]."""
    check(_l.lib().ti_moe_permute(ptr(h), g.T, h.stride(0), ptr(g.ids), ptr(g.pos), ptr(g.first), ptr(g.slot), ptr(xs), g.E, g.top,
                                  xs.shape[0], _f32(h), stream()), "ti_moe_permute")


def gemm_grouped(W: "LinearW", E: int, x, g: TokenGroups, *, out, epi=GEPI_STORE, ex=None):
    """y[r] = x[r] W_e^T for the rows of every token tile; W holds the E matrices one after the other.  x: bf16 rows, or
    their limb planes for int8 matrices."""
    N, nt, tab = W.N // E, W.n_tiles // E, (ptr(g.tiles), ptr(g.num_tiles), g.tiles.shape[1], g.tile)
    assert W.N == N * E and N % 8 == 0
    ldo = 0 if out is None else out.stride(0)
    if W.wt == W_BF16:
        check(_l.lib().ti_gemm_grouped_bf16(ptr(W.tiles), E, nt, N, W.K, ptr(x), x.shape[0], *tab, ptr(out), ldo, epi, status_ptr(),
                                            _ref(ex), stream()), "ti_gemm_grouped_bf16")
    else:
        check(_l.lib().ti_gemm_grouped_w8a16(ptr(W.tiles), ptr(W.scale), E, nt, N, W.K, ptr(x.hi), ptr(x.lo), ptr(x.scale), x.M, *tab,
                                             ptr(out), ldo, epi, status_ptr(), _ref(ex), stream()), "ti_gemm_grouped_w8a16")
