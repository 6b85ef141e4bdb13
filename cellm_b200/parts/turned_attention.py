"""Attention inside chunks of positions whose queries and keys are turned first and normed afterwards.

    q, k, v = W h                                            (no biases)
    q, k: the first `rotary_dim` entries of every head turn by pos * f_i (the position part; its amplitude multiplies cos
          and sin), then every head is divided by its own root mean square over all its entries, without a weight
          (`unit_eps`; None: not)
    softmax of (q . k) * scale over the keys j <= i with floor(j / chunk) = floor(i / chunk), chunks counted from position 0
          of the sequence (chunk 0: every earlier key); query head h uses key/value head floor(h / (heads / kv_heads))
    out = W_o (heads side by side)

Keys are cached turned and normed. A layer may read the keys and values of another item of the run order (`reads` True):
it has queries of its own only, and a chunk of its own. The pages of the item that is read keep what every reader needs
(`kept_chunk` or `kept_window`, the same for the reader and the item it reads).

Rows of the cache are kept `width` wide, zeros behind a head's own entries, where that brings keys and values to a width
the tensor-core kernels are built for (32, 64, 96 or 128).

Kernels: one product for q | k | v with 32-bit sums, `turned_attn_prep` (rotation, norm, cache write), the attention itself
(bfloat16: tcgen05 for prompt portions that fill its tiles with heads of 64, else the paged mma.sync flash kernel; 32-bit
and heads wider than 128: the plain kernel), the output product. Scores, softmax, angles and norms are 32-bit."""
from __future__ import annotations

import torch

from ..config.errors import ConfigError
from ..config.plan import PartSpec
from .base import CacheBinding, Mixer, PagedKV, StepContext, TensorSpec
from .linear import Linear, stack_rows
from .registry import part_class, register_mixer

# Tests turn the tensor-core attention off to compare it with the plain kernel on the same cache, and the tcgen05 kernel
# off to compare it with the mma.sync one.
OPTIONS = {"tensor_cores": True, "tcgen05": True}

WIDTHS = (32, 64, 96, 128)


def row_width(hd: int, vd: int) -> int:
    """The width of a cached row of keys and values that the tensor-core kernels take, or 0 (rows as wide as the heads)."""
    return next((w for w in WIDTHS if w >= max(hd, vd)), 0)


class TurnedAttentionMixer(Mixer):
    graph_safe = True
    can_read_foreign_cache = True

    """params: hidden_size, num_heads, num_kv_heads, head_dim, value_dim (default head_dim), scale, chunk (default 0), unit_eps
    (default None), position (PartSpec of a rotation, or None), reads (default False: keys and values of its own),
    kept_chunk (default chunk) and kept_window (default 0): what the pages keep, out_dtype32 (default False).
    weights: q_proj [nh*hd, H], out_proj [H, nh*vd]; k_proj [nkv*hd, H] and v_proj [nkv*vd, H] unless it reads another's."""

    @classmethod
    def _sizes(cls, params):
        nh, nkv, hd = int(params["num_heads"]), int(params["num_kv_heads"]), int(params["head_dim"])
        return nh, nkv, hd, int(params.get("value_dim") or hd)

    @classmethod
    def weight_specs(cls, params):
        H = params["hidden_size"]
        nh, nkv, hd, vd = cls._sizes(params)
        specs = {"q_proj": TensorSpec((nh * hd, H), "linear"), "out_proj": TensorSpec((H, nh * vd), "linear")}
        if not params.get("reads"):
            specs.update(k_proj=TensorSpec((nkv * hd, H), "linear"), v_proj=TensorSpec((nkv * vd, H), "linear"))
        return specs

    @classmethod
    def cache_need(cls, params):
        nh, nkv, hd, vd = cls._sizes(params)
        window = int(params.get("kept_window") or 0)
        chunk = 0 if window else int(params.get("kept_chunk", params.get("chunk") or 0) or 0)
        w = row_width(hd, vd)
        if w:
            return PagedKV(nkv, w, window, chunk=chunk)
        return PagedKV(nkv, hd, window, value_dim=vd if vd != hd else 0, chunk=chunk)

    def __init__(self, params: dict, weights: dict, dtype: torch.dtype):
        self.H = int(params["hidden_size"])
        self.nh, self.nkv, self.hd, self.vd = self._sizes(params)
        if self.nh % self.nkv:
            raise ConfigError(f"turned_attention: {self.nh} heads are not a multiple of {self.nkv} key/value heads")
        self.scale, self.chunk = float(params["scale"]), int(params.get("chunk") or 0)
        self.unit_eps = params.get("unit_eps")
        self.reads, self.dtype = bool(params.get("reads")), dtype
        self.out32 = bool(params.get("out_dtype32", False))
        width = row_width(self.hd, self.vd)
        self.row_k, self.row_v = (width, width) if width else (self.hd, self.vd)
        mats = [weights["q_proj"]] + ([] if self.reads else [weights["k_proj"], weights["v_proj"]])
        self.qkv = Linear(stack_rows(*mats), dtype)
        out_w = weights["out_proj"]
        if self.row_v != self.vd:       # zero columns where the widened heads' values are zero
            wide = torch.zeros((self.H, self.nh, self.row_v), dtype=out_w.dtype, device=out_w.device)
            wide[:, :, :self.vd] = out_w.reshape(self.H, self.nh, self.vd)
            out_w = wide.reshape(self.H, self.nh * self.row_v)
        self.out_proj = Linear(out_w, dtype)
        dev = weights["q_proj"].device
        pos: PartSpec | None = params.get("position")
        self.position = part_class("position", pos.kind)(pos.params, dev) if pos is not None else None
        self.rot, self.interleaved, self.freq, self.amp = 0, False, None, 1.0
        if self.position is not None:
            r = self.position.rotation(amplitude=True)
            if r is None:
                raise ConfigError("turned_attention: the position encoding must be a rotation")
            self.rot, self.interleaved, self.freq, self.amp = int(r[0]), bool(r[1]), r[2], float(self.position.amplitude)

    def _tcgen05(self, ctx: StepContext, cache: CacheBinding) -> bool:
        from ..ops._state import sm_count
        from ..ops.attention import attention_tc_fills, attention_tc_supports
        from ..runtime.program import OPTIONS as RUN
        if not OPTIONS["tcgen05"] or self.scale <= 0 or not attention_tc_supports(self.row_k, self.nh, self.nkv, cache.page_size):
            return False
        return attention_tc_fills(ctx.q_lens, self.nh, self.nkv, sm_count(ctx.device), RUN["attention_tc_min_ctas"], RUN["attention_tc_min_fill"])

    def forward(self, x: torch.Tensor, ctx: StepContext, cache: CacheBinding) -> torch.Tensor:
        from .. import ops
        proj = self.qkv(x, out_dtype=torch.float32)
        q = ops.turned_attn_prep(proj, self.freq, self.rot, self.interleaved, self.amp, self.unit_eps, ctx, cache, self.nh,
                                 0 if self.reads else self.nkv, self.hd, self.vd, self.row_k, self.dtype)
        if self.dtype == torch.bfloat16 and self.row_k == self.row_v and self.row_k in WIDTHS and OPTIONS["tensor_cores"] and self.scale > 0:
            if self._tcgen05(ctx, cache):
                o = ops.attention_tc_chunked(q, cache, ctx, self.nh, self.nkv, self.scale, self.chunk)
            else:
                o = ops.attention_flash_chunked(q, cache, ctx, self.nh, self.nkv, self.row_k, self.scale, self.chunk)
        else:
            o = ops.attention_plain_chunked(q, cache, ctx, self.nh, self.nkv, self.row_k, self.row_v, self.scale, self.chunk)
        return self.out_proj(o, out_dtype=torch.float32 if self.out32 else None)


register_mixer("turned_attention", TurnedAttentionMixer)
