"""The op records of the native executor (csrc/runtime/executor.h) as ctypes
structures, and what a part's emit() appends them to.

A part describes itself to the executor with one record: its kind and a
parameter struct that points at its weights. A part without a native record
emits a Python record instead, and the executor calls back into the
interpreter for that part alone.
"""
from __future__ import annotations

import ctypes
from ctypes import POINTER, Structure, c_double, c_longlong, c_void_p
from typing import Optional

import torch

from ..ops import _lib as klib

I64, F64, PTR = c_longlong, c_double, c_void_p

# record kinds, in the order of the executor's OpKind
(EMBED, RMS_NORM, SHORT_CONV, ATTENTION, SWIGLU, HEAD, PYTHON, LINEAR, ATTEND,
 READ_STREAM, GATED_NORM_ADD, MINGRU, LATENT_ATTENTION, GATED_MLP, ROUTED_MLP, RESULT_NORM) = range(16)


class ExecLinear(Structure):
    _fields_ = [("w", PTR), ("N", I64), ("K", I64), ("ldw", I64), ("dtype", I64), ("tc_ok", I64)]


class ExecOp(Structure):
    _fields_ = [("kind", I64), ("params", PTR)]


class EmbedParams(Structure):
    _fields_ = [("table", PTR), ("dtype", I64), ("scale", F64), ("pos_table", PTR), ("max_pos", I64)]


class RmsNormParams(Structure):
    _fields_ = [("w", PTR), ("dtype", I64), ("eps", F64), ("groups", I64)]


class ShortConvParams(Structure):
    _fields_ = [("in_proj", ExecLinear), ("out_proj", ExecLinear), ("in_proj_tiled", PTR), ("tiled_rows", I64),
                ("taps", PTR), ("bias", PTR), ("taps_dtype", I64), ("n_taps", I64)]


class AttentionParams(Structure):
    _fields_ = [("qkv", ExecLinear), ("out_proj", ExecLinear), ("nh", I64), ("nkv", I64), ("hd", I64), ("window", I64),
                ("scale", F64), ("q_norm_w", PTR), ("k_norm_w", PTR), ("qk_dtype", I64), ("qk_eps", F64),
                ("rot", I64), ("interleaved", I64), ("inv_freq", PTR), ("hdv", I64), ("norm_whole", I64),
                ("temp_coef", F64), ("temp_every", I64), ("pad", I64)]


class SwiGLUParams(Structure):
    _fields_ = [("gate_up", ExecLinear), ("down", ExecLinear), ("ff", I64), ("fused", I64)]


class HeadParams(Structure):
    _fields_ = [("w", ExecLinear), ("soft_cap", F64)]


class PythonParams(Structure):
    _fields_ = [("token", I64)]


class LinearParams(Structure):
    _fields_ = [("w", ExecLinear), ("lda", I64), ("out_dtype", I64)]


class ReadStreamParams(Structure):
    _fields_ = [("reserved", I64)]


class GatedNormAddParams(Structure):
    _fields_ = [("gate", ExecLinear), ("gate_bias", PTR), ("w", PTR), ("w_dtype", I64), ("groups", I64), ("eps", F64), ("stacked", I64)]


class MinGruParams(Structure):
    _fields_ = [("in_proj", ExecLinear), ("out_proj", ExecLinear), ("bz", PTR), ("bx", PTR), ("b_dtype", I64), ("width", I64), ("extra", I64)]


class LatentAttentionParams(Structure):
    _fields_ = [("in_proj", ExecLinear), ("out_proj", ExecLinear), ("absorb_k", PTR), ("expand_v", PTR),
                ("heads", I64), ("dim", I64), ("rot_dim", I64), ("vdim", I64), ("rank", I64), ("scale", F64),
                ("c_norm_w", PTR), ("c_norm_dtype", I64), ("eps", F64), ("rot", I64), ("inv_freq", PTR), ("extra", I64),
                ("interleaved", I64), ("window", I64), ("sinks", PTR), ("amplitude", F64), ("q_up", ExecLinear), ("q_norm_w", PTR),
                ("q_rank", I64), ("gate", I64), ("kv_up", ExecLinear)]


class GatedMlpParams(Structure):
    _fields_ = [("gate_up", ExecLinear), ("down", ExecLinear), ("bg", PTR), ("bu", PTR), ("bd", PTR), ("b_dtype", I64),
                ("ff", I64), ("act", I64), ("extra", I64), ("fused", I64), ("out32", I64), ("limit", F64), ("slope", F64)]


class RoutedMlpParams(Structure):
    _fields_ = [("up", ExecLinear), ("down", ExecLinear), ("router", ExecLinear), ("correction", PTR), ("c_dtype", I64),
                ("experts", I64), ("top", I64), ("n_groups", I64), ("keep", I64), ("scale", F64), ("ff", I64), ("act", I64),
                ("shared_up", ExecLinear), ("shared_down", ExecLinear), ("shared_ff", I64), ("shared_gate", I64),
                ("gated", I64), ("softmax", I64), ("out32", I64), ("gate_kind", I64), ("limit", F64), ("shared_limit", F64), ("slope", F64)]


class ResultNormParams(Structure):
    _fields_ = [("w", PTR), ("w_dtype", I64), ("eps", F64)]


class ExecOps(Structure):
    _fields_ = [("n", I64), ("ops", POINTER(ExecOp))]


class ExecRegs(Structure):
    _fields_ = [("x", PTR), ("pending", PTR), ("y", PTR), ("logits", PTR), ("phase", I64), ("item", I64)]


PythonOpFn = ctypes.CFUNCTYPE(c_longlong, c_longlong, POINTER(ExecRegs))

# the kernel libraries' entry points in the order of the executor's table (ExecFn)
ENTRY_POINTS = [("kernels_common", "cellm_embed"), ("kernels_common", "cellm_add_rmsnorm"), ("kernels_common", "cellm_residual_add"),
                ("kernels_common", "cellm_swiglu"), ("kernels_common", "cellm_short_conv"), ("kernels_common", "cellm_qk_norm_rope"),
                ("kernels_common", "cellm_attention_plain"), ("gemm_plain", "cellm_gemm_plain"),
                ("attention_decode", "cellm_attention_decode"), ("attention_tc", "cellm_attention_tc"),
                ("attention_flash", "cellm_attention_flash"), ("gemm_tcgen05", "cellm_gemm_tcgen05"),
                ("gemm_tcgen05", "cellm_gemm_conv_tcgen05"), ("gemm_tcgen05", "cellm_gemm_rope_tcgen05"),
                ("kernels_common", "cellm_gated_norm_add"), ("kernels_common", "cellm_stream_cast"),
                ("kernels_common", "cellm_mingru_scan"), ("kernels_common", "cellm_latent_prep"),
                ("kernels_common", "cellm_head_product"), ("kernels_common", "cellm_gated_act"), ("kernels_common", "cellm_bias_add"),
                ("attention_latent", "cellm_attention_latent"), ("attention_latent", "cellm_head_product_mma"),
                ("kernels_common", "cellm_embed_pos"), ("kernels_common", "cellm_attn_prep"),
                ("kernels_common", "cellm_attention_plain_wide"), ("kernels_common", "cellm_route"),
                ("kernels_common", "cellm_experts_rowwise"), ("kernels_common", "cellm_activation"),
                ("kernels_common", "cellm_add2_rmsnorm"), ("kernels_common", "cellm_moe_sort"), ("kernels_common", "cellm_moe_gather"),
                ("kernels_common", "cellm_moe_combine"), ("gemm_tcgen05", "cellm_gemm_grouped_tcgen05"),
                ("kernels_common", "cellm_attention_plain_masked"), ("kernels_common", "cellm_route_softmax"),
                ("kernels_common", "cellm_experts_gated_rowwise"), ("kernels_common", "cellm_moe_combine32"),
                ("gemm_tcgen05", "cellm_gemm_gated_tcgen05"), ("gemm_tcgen05", "cellm_gemm_grouped_gated_tcgen05"),
                ("kernels_common", "cellm_clamped_gate_act"), ("kernels_common", "cellm_norm_add_norm"), ("kernels_common", "cellm_soft_cap"),
                ("kernels_common", "cellm_route_softmax_all"), ("attention_expanded", "cellm_latent_rows"),
                ("attention_expanded", "cellm_attention_expanded"), ("attention_expanded", "cellm_attention_expanded_supports")]
# libraries a model whose activations are 32-bit never calls into (they need not be compiled for it)
BF16_ONLY_LIBRARIES = ("attention_decode", "attention_tc", "attention_flash", "gemm_tcgen05", "attention_latent", "attention_expanded")
# libraries that only records of these kinds reach (a program without such a record need not have them compiled)
LIBRARY_USERS = {"attention_decode": (ATTENTION, ATTEND), "attention_tc": (ATTENTION, ATTEND), "attention_flash": (ATTENTION, ATTEND),
                 "attention_latent": (LATENT_ATTENTION,), "attention_expanded": (LATENT_ATTENTION,)}


class ExecProgram(Structure):
    _fields_ = [("n_layers", I64), ("n_order", I64), ("H", I64), ("V", I64), ("act_dtype", I64),
                ("sms", I64), ("static_flag", I64), ("max_counters", I64), ("fused_conv", I64), ("fused_rope", I64),
                ("latent_tc", I64), ("latent_expand", I64), ("grouped_min_tokens", I64), ("tc_min_ctas", I64), ("tc_min_fill", F64),
                ("prologue", ExecOps), ("epilogue", ExecOps), ("layers", POINTER(ExecOps)), ("order", POINTER(I64)),
                ("python", PythonOpFn), ("fns", PTR * len(ENTRY_POINTS))]


class ExecItem(Structure):
    _fields_ = [("k", PTR), ("v", PTR), ("block_table", PTR), ("bt_stride", I64), ("num_pages", I64), ("page_size", I64),
                ("writes", I64), ("state", PTR), ("slot_stride", I64), ("n_slots", I64)]


class ExecStep(Structure):
    _fields_ = [("T", I64), ("B", I64), ("R", I64), ("max_q_len", I64), ("max_total_len", I64), ("n_order", I64),
                ("ids", PTR), ("positions", PTR), ("seq_of_token", PTR), ("cu_seqlens", PTR), ("ctx_lens", PTR),
                ("slot_ids", PTR), ("rows", PTR), ("q_lens", POINTER(I64)), ("host_ctx_lens", POINTER(I64)), ("items", POINTER(ExecItem)),
                ("arena", PTR), ("arena_bytes", I64), ("logits", PTR), ("err", PTR), ("stream", PTR),
                ("gemm_ws", PTR), ("gemm_ws_floats", I64), ("attn_ws", PTR), ("attn_ws_floats", I64), ("counters", PTR),
                ("launches", I64), ("calls", I64 * len(ENTRY_POINTS))]


# in the order cellm_exec_sizeof() numbers them
LAYOUT_CHECKED = (ExecLinear, ExecOp, ExecProgram, ExecItem, ExecStep, ExecRegs, EmbedParams, RmsNormParams, ShortConvParams,
                  AttentionParams, SwiGLUParams, HeadParams, PythonParams, ExecOps, LinearParams, ReadStreamParams, GatedNormAddParams,
                  MinGruParams, LatentAttentionParams, GatedMlpParams, RoutedMlpParams, ResultNormParams)


def ptr(t: Optional[torch.Tensor]):
    return None if t is None else t.data_ptr()


def linear(weight: torch.Tensor, rows: Optional[int] = None) -> ExecLinear:
    """A weight matrix [N, K] as the executor's products read it (`rows`: only its first rows)."""
    w = weight
    ok = w.stride(1) == 1 and w.stride(0) % 8 == 0 and w.data_ptr() % 16 == 0
    return ExecLinear(w.data_ptr(), rows if rows is not None else w.shape[0], w.shape[1], w.stride(0), klib.tag(w), int(ok))


class Record:
    """One op record with what it points to kept alive."""

    def __init__(self, kind: int, params: Structure, keep=(), part=None, role: str = ""):
        self.kind, self.params, self.keep, self.part, self.role = kind, params, list(keep), part, role
        self.op = ExecOp(kind, ctypes.cast(ctypes.pointer(params), c_void_p).value)


class Emitter:
    """What a part's emit() appends its records to. `act_dtype` is the element type of the activations the records
    will work on: a part whose weights do not fit it emits a Python record (`python(role, part)`) instead."""

    def __init__(self, act_dtype: torch.dtype, tokens: list):
        self.act_dtype = act_dtype
        self.records: list[Record] = []
        self._tokens = tokens          # the program's list of (role, part) that Python records name by index

    def native(self, kind: int, params: Structure, keep=(), part=None) -> None:
        self.records.append(Record(kind, params, keep, part))

    def python(self, role: str, part) -> None:
        """`role`: "embedding", "norm", "mixer", "feed_forward", "block" or "head": which forward() the executor's
        call-back runs on the registers (see Program._python_op)."""
        self._tokens.append((role, part))
        self.records.append(Record(PYTHON, PythonParams(len(self._tokens) - 1), part=part, role=role))

    def fits(self, *weights: torch.Tensor) -> bool:
        """Whether matrices kept in these element types can be multiplied with the activations natively."""
        return all(w.dtype == self.act_dtype for w in weights)
