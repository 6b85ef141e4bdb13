"""ctypes bindings to the compiled kernels. A missing or unbuildable library
raises at first use; there is no fallback to another implementation."""
from __future__ import annotations

import ctypes
from ctypes import c_float, c_int, c_longlong, c_void_p

import torch

from ..csrc import build as _build

P, I, L, F = c_void_p, c_int, c_longlong, c_float

DTYPE_TAG = {torch.float32: 0, torch.bfloat16: 1}

_ERRORS = {-1: "unsupported element type", -2: "a size this kernel does not take",
           -3: "a pointer or stride breaks an alignment rule", -4: "missing or contradictory argument"}

_SIGNATURES = {
    "kernels_common": {
        "cellm_embed": [P, P, I, P, I, I, I, F, P, P],
        "cellm_embed_pos": [P, P, I, P, P, P, I, I, I, I, F, P, P],
        "cellm_upload": [P, P, L, P],
        "cellm_add_rmsnorm": [P, P, P, I, P, P, I, I, I, F, I, P],
        "cellm_add2_rmsnorm": [P, P, P, P, I, P, P, I, I, I, F, I, P],
        "cellm_residual_add": [P, P, L, I, P],
        "cellm_swiglu": [P, P, I, I, I, I, P],
        "cellm_short_conv": [P, P, P, P, I, P, L, P, P, P, I, I, I, I, I, I, I, P, P],
        "cellm_qk_norm_rope": [P, P, L, P, P, I, F, P, P, P, I, P, P, I, I, I, I, I, I, I, I, P, I, P, P],
        "cellm_attention_plain": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, F, I, I, P, P],
        "cellm_gated_norm_add": [P, P, P, P, L, I, P, P, I, P, I, I, I, F, I, P],
        "cellm_stream_cast": [P, P, L, I, P],
        "cellm_mingru_scan": [P, P, L, I, P, P, I, P, L, P, P, I, I, I, I, I, I, P, P],
        "cellm_latent_prep": [P, P, L, P, P, P, L, I, P, L, I, P, I, I, P, I, F, P, P, P, I, P, I, I, I, I, I, I, I, I, I, P, F, I, I, P, P],
        "cellm_head_product": [P, L, L, P, L, L, P, I, I, I, I, I, P],
        "cellm_gated_act": [P, P, L, P, P, I, I, I, I, I, I, P],
        "cellm_bias_add": [P, P, P, I, I, I, I, P],
        "cellm_attn_prep": [P, P, L, P, P, I, F, I, F, I, P, P, P, I, P, P, I, I, I, I, I, I, I, I, I, I, P, P],
        "cellm_attention_plain_wide": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, F, I, I, P, P],
        "cellm_route": [P, P, P, P, L, P, I, I, I, I, I, I, F, I, P],
        "cellm_experts_rowwise": [P, P, P, P, L, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, P],
        "cellm_activation": [P, P, L, I, I, I, I, P],
        "cellm_moe_sort": [P, P, P, P, I, I, I, P],
        "cellm_moe_gather": [P, P, L, P, P, I, I, I, P],
        "cellm_moe_combine": [P, P, P, P, P, P, I, I, I, P],
        "cellm_argmax": [P, P, I, I, P, P],
        "cellm_take_pending_tokens": [P, P, P, P, I, I, P, P],
        "cellm_keep_last_tokens": [P, P, P, I, I, P],
        "cellm_sample": [P, P, I, I, P, P, P, P, P, I, I, P, P],
        "cellm_embed_pairs": [P, P, I, P, P, L, L, L, P, L, I, P, P, P, P, I, I, I, F, P, P],
        "cellm_norm_pair": [P, P, P, P, P, I, I, I, F, I, P],
        "cellm_scaled_add2": [P, P, P, F, L, I, P],
        "cellm_pair_norm_mean": [P, P, P, P, P, I, I, F, I, P],
        "cellm_conv_state_update": [P, L, I, P, P, P, L, I, P, I, I, I, P, P],
        "cellm_sink_attn_prep": [P, P, P, P, L, I, P, P, I, P, L, I, P, P, F, P, I, P, I, P, P, P, P, P, I, I, I, I, I, I, I, I, P, I, P, P],
        "cellm_attention_plain_masked": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, I, P, F, I, P, L, I, P, P],
        "cellm_attention_plain_sink": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, F, I, P, P, I, I, P, P],
        "cellm_hgrn2_scan": [P, P, L, I, P, L, I, I, I, P, P, P, P, I, I, I, I, I, P, P],
        "cellm_delta_prep": [P, P, P, P, P, L, I, I, P, I, P, L, I, P, L, P, P, P, P, P, I, I, I, I, I, F, P, P],
        "cellm_delta_scan": [P, P, L, I, P, P, P, P, P, P, I, I, I, I, I, P, P],
        "cellm_head_norm_gate": [P, P, P, P, L, I, I, I, F, I, I, P],
        "cellm_gdelta_prep": [P, P, L, I, I, P, L, P, P, F, F, I, I, I, P],
        "cellm_gdelta_scan": [P, P, L, I, P, L, I, I, I, P, P, P, I, I, I, I, P, P],
        "cellm_add_scaled_norm": [P, P, P, F, P, F, I, P, P, P, I, I, I, F, I, I, P],
        "cellm_stream_add_rows": [P, P, I, P, I, F, P, I, I, P, P],
        "cellm_token_gate_mul": [P, P, L, P, L, I, I, P, I, I, I, I, I, P, P],
        "cellm_scaled_rms_add": [P, P, P, F, I, I, F, P],
        "cellm_weighted_sum2": [P, P, F, P, F, L, I, P],
        "cellm_xielu": [P, P, L, I, I, P, I, P],
        "cellm_head_gate_mul": [P, P, L, I, I, I, I, P],
        "cellm_route_softmax": [P, P, P, P, L, P, I, I, I, I, F, I, P],
        "cellm_experts_gated_rowwise": [P, P, P, P, L, P, P, P, P, P, P, P, I, I, I, I, I, I, I, F, F, F, I, I, P],
        "cellm_norm_add_norm": [P, P, P, F, P, I, P, P, I, I, F, I, P],
        "cellm_soft_cap": [P, L, F, P],
        "cellm_route_softmax_all": [P, P, P, P, L, P, I, I, I, I, I, I, F, I, P],
        "cellm_moe_combine32": [P, P, P, P, P, P, I, I, I, P],
        "cellm_clamped_gate_act": [P, P, L, I, I, F, F, I, P],
        "cellm_embed_norm": [P, P, I, P, P, I, I, I, F, F, P, P],
        "cellm_post_norm": [P, P, P, I, F, P, I, I, F, I, P],
        "cellm_turned_attn_prep": [P, P, P, P, L, P, I, I, F, I, F, P, P, P, I, I, I, I, I, I, I, I, I, I, I, P, P],
        "cellm_attention_plain_chunked": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, F, I, I, P, P],
        "cellm_decay_scan": [P, P, L, I, P, L, P, L, P, L, P, L, P, L, P, P, I, I, I, I, I, I, P, P],
        "cellm_rotate_heads": [P, L, I, I, I, I, I, P, F, P, I, P],
        "cellm_ssd_prep": [P, P, P, P, P, L, I, I, I, P, I, P, P, L, I, P, P, P, P, P, I, I, P, P],
        "cellm_gated_group_norm": [P, P, P, L, P, P, L, P, I, I, I, I, F, I, P],
        "cellm_head_norm_silu": [P, P, P, L, I, I, I, F, I, P],
    },
    "gemm_plain": {
        "cellm_gemm_plain": [P, P, P, I, I, I, L, L, L, I, I, P],
    },
    "attention_decode": {
        "cellm_attention_decode": [P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, F, I, I, P, P],
    },
    "attention_tc": {
        "cellm_attention_tc": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, P, P],
        "cellm_attention_tc_supports": [I, I, I, I],
        "cellm_attention_tc_chunked": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, P, P],
        "cellm_attention_tc_gated": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, P, P, L, P, P],
    },
    "attention_flash": {
        "cellm_attention_flash": [P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, I, I, P, P],
        "cellm_attention_flash_supports": [I],
        "cellm_attention_flash_sink": [P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, I, I, P, P, I, P, P, P],
        "cellm_attention_flash_chunked": [P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, I, I, P, P],
        "cellm_attention_flash_masked": [P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, I, I, I, P, P, L, P, P],
    },
    "decay_chunks": {
        "cellm_decay_chunks": [P, P, L, I, P, L, P, L, P, L, P, L, P, L, P, P, I, I, I, I, I, I, I, P, P, P, P],
        "cellm_decay_chunks_supports": [I, I],
    },
    "attention_expanded": {
        "cellm_latent_rows": [P, P, P, P, P, I, I, I, I, I, I, I, P, P],
        "cellm_attention_expanded": [P, P, L, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, P, P, P, P],
        "cellm_attention_expanded_supports": [I, I, I, I, I],
    },
    "attention_latent": {
        "cellm_attention_latent": [P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, I, P, P, P, P],
        "cellm_attention_latent_supports": [I, I],
        "cellm_head_product_mma": [P, L, L, P, L, L, P, I, I, I, I, P],
    },
    "gemm_tcgen05": {
        "cellm_gemm_tcgen05": [P, P, P, I, I, I, L, L, L, I, I, I, I, I, P, P, P, P],
        "cellm_gemm_grouped_tcgen05": [P, P, P, I, I, I, I, L, L, L, I, P, I, P, P],
        "cellm_gemm_gated_tcgen05": [P, P, P, I, I, I, L, L, L, I, I, I, I, F, F, I, P, P, P, P],
        "cellm_gemm_grouped_gated_tcgen05": [P, P, P, I, I, I, I, L, L, L, I, P, I, F, F, P, P],
        "cellm_gemm_xielu_tcgen05": [P, P, P, I, I, I, L, L, L, I, P, P, P],
        "cellm_gemm_conv_tcgen05": [P, P, P, I, I, I, L, L, I, I, I, P, P, I, P, L, P, I, I, P, P],
        "cellm_gemm_rope_tcgen05": [P, P, P, I, I, L, L, I, I, P, P, F, P, P, I, P, P, I, I, I, I, P, I, P, P],
    },
}

_funcs: dict[str, ctypes._CFuncPtr] = {}

# Kernels launched through these bindings since the process began: every entry
# point launches one kernel unless listed here.
LAUNCHES = [0]
_KERNELS_PER_CALL = {}


def count_launch(n: int = 1) -> None:
    LAUNCHES[0] += n


def register_signatures(library: str, signatures: dict) -> None:
    _SIGNATURES.setdefault(library, {}).update(signatures)


def fn(library: str, name: str):
    f = _funcs.get(name)
    if f is None:
        lib = _build.load(library)
        f = getattr(lib, name)
        f.argtypes = _SIGNATURES[library][name]
        f.restype = c_int
        _funcs[name] = f
    return f


def check(code: int, name: str) -> None:
    if code == 0:
        LAUNCHES[0] += _KERNELS_PER_CALL.get("cellm_" + name, 1)
        return
    if code < 0:
        raise ValueError(f"{name}: refused: {_ERRORS.get(code, code)}")
    raise RuntimeError(f"{name}: CUDA error {code} at launch")


def ptr(t):
    return None if t is None else t.data_ptr()


def tag(t_or_dtype) -> int:
    dt = t_or_dtype if isinstance(t_or_dtype, torch.dtype) else t_or_dtype.dtype
    try:
        return DTYPE_TAG[dt]
    except KeyError:
        raise ValueError(f"element type {dt} is not supported by the kernels") from None


# The raw handle of the current stream, asked from torch's C layer where that entry point exists: the Python
# wrapper (torch.cuda.current_stream) costs about 8 us a call, which every launch would pay.
_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)


def stream_of(t: torch.Tensor) -> int:
    if _raw_stream is not None:
        return _raw_stream(t.device.index or 0)
    return torch.cuda.current_stream(t.device).cuda_stream


def require_cuda(*tensors) -> None:
    for t in tensors:
        if t is not None and (not t.is_cuda or not t.is_contiguous()):
            raise ValueError("kernel arguments must be contiguous CUDA tensors "
                             f"(got device={t.device}, contiguous={t.is_contiguous()})")
