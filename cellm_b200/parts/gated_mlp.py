"""Gated feed-forward in its general form: W_down (act(W_gate h + b_gate) * (W_up h + b_up)) + b_down, with act
"silu" or "gelu_tanh" (0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))) and optional biases. Gate and up are
stacked so that one product yields both; they stay 32-bit until act(g) * u is formed.

"clamped" joins the two otherwise: g' sigmoid(slope g') (u' + 1) with g' = min(g, limit) and u' = clamp(u, -limit, limit). Under
bfloat16 it is formed in the first product's epilogue: gate and up rows are then kept in blocks of 64 (the width padded to
a multiple of 64 with zero rows, whose middles are zero)."""
from __future__ import annotations

import torch

from ..config.errors import ConfigError
from .base import FeedForward, StepContext, TensorSpec
from .linear import Linear, stack_rows
from .registry import register_feed_forward

ACTIVATIONS = {"silu": 0, "gelu_tanh": 1, "clamped": 2}
BLOCK = 64      # rows of a block of gate or up rows in the layout of the products whose epilogue joins the two


def blocked_gate_up(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """gate, up [n, K] as [2 n', K] in blocks of 64 gate rows followed by their 64 up rows, n' = n rounded up to whole blocks
    (zero rows behind n)."""
    n, K = gate.shape
    wide = -(-n // BLOCK) * BLOCK
    both = torch.zeros((2, wide, K), dtype=gate.dtype if gate.dtype == up.dtype else torch.float32, device=gate.device)
    both[0, :n], both[1, :n] = gate, up
    return both.reshape(2, wide // BLOCK, BLOCK, K).transpose(0, 1).reshape(2 * wide, K).contiguous()


def widened_columns(down: torch.Tensor) -> torch.Tensor:
    """down [H, n] with zero columns up to a multiple of 64."""
    H, n = down.shape
    wide = -(-n // BLOCK) * BLOCK
    if wide == n:
        return down.contiguous()
    out = torch.zeros((H, wide), dtype=down.dtype, device=down.device)
    out[:, :n] = down
    return out


class GatedMLP(FeedForward):
    graph_safe = True

    """params: hidden_size, ff_dim, activation, bias, limit (default none) and slope (default 1) for "clamped", out_dtype32
    (default False: the result in the activations' type). weights: gate, up [ff, H]; down [H, ff];
    gate_bias, up_bias [ff], down_bias [H] if bias."""

    @classmethod
    def weight_specs(cls, params):
        H, ff = params["hidden_size"], params["ff_dim"]
        specs = {"gate": TensorSpec((ff, H), "linear"), "up": TensorSpec((ff, H), "linear"), "down": TensorSpec((H, ff), "linear")}
        if params.get("bias"):
            specs.update(gate_bias=TensorSpec((ff,), "bias"), up_bias=TensorSpec((ff,), "bias"), down_bias=TensorSpec((H,), "bias"))
        return specs

    def __init__(self, params: dict, weights: dict, dtype: torch.dtype):
        self.H, self.ff, self.dtype = int(params["hidden_size"]), int(params["ff_dim"]), dtype
        self.activation = params.get("activation", "silu")
        if self.activation not in ACTIVATIONS:
            raise ConfigError(f"gated_mlp: activation {self.activation!r}; known: {sorted(ACTIVATIONS)}")
        limit = params.get("limit")
        self.limit, self.slope = float("inf") if limit is None else float(limit), float(params.get("slope", 1.0))
        self.out32 = bool(params.get("out_dtype32", False))
        if self.activation == "clamped" and params.get("bias"):
            raise ConfigError("gated_mlp: the clamped gate has no biases")
        self.fused = (self.activation == "clamped" and dtype == torch.bfloat16 and self.H % 8 == 0
                      and all(weights[k].dtype == torch.bfloat16 for k in ("gate", "up", "down")))
        if self.fused:
            self.gate_up, self.down = Linear(blocked_gate_up(weights["gate"], weights["up"]), dtype), Linear(widened_columns(weights["down"]), dtype)
            self.ff = self.down.in_features
        else:
            self.gate_up = Linear(stack_rows(weights["gate"], weights["up"]), dtype)
            self.down = Linear(weights["down"], dtype)
        self.bg = self.bu = self.bd = None
        if params.get("bias"):
            self.bg = weights["gate_bias"].contiguous()
            self.bu = weights["up_bias"].to(self.bg.dtype).contiguous()
            self.bd = weights["down_bias"].to(self.bg.dtype).contiguous()
        self.extra = 0
        self._record = None

    def stack_behind_input(self, weight: torch.Tensor) -> bool:
        if self._record is not None or self.extra or self.activation == "clamped" or weight.dtype != self.gate_up.weight.dtype or weight.shape[1] != self.H:
            return False
        self.gate_up = Linear(stack_rows(self.gate_up.weight, weight), self.dtype)
        self.extra = int(weight.shape[0])
        return True

    def stacked_rows(self) -> torch.Tensor:
        return self.gate_up.weight[self.gate_up.weight.shape[0] - self.extra:]

    def record(self):
        from ..ops._lib import tag
        from ..runtime import records as R
        if self._record is None and self.gate_up.weight.dtype == self.dtype == self.down.weight.dtype:
            p = R.GatedMlpParams(R.linear(self.gate_up.weight), R.linear(self.down.weight), R.ptr(self.bg), R.ptr(self.bu),
                                 R.ptr(self.bd), tag(self.bg) if self.bg is not None else tag(self.dtype), self.ff,
                                 ACTIVATIONS[self.activation], self.extra, int(self.fused), int(self.out32), self.limit, self.slope)
            self._record = R.Record(R.GATED_MLP, p, part=self)
        return self._record

    def emit(self, emitter) -> None:
        rec = self.record()
        if rec is None or self.out32:       # the executor's registers hold results in the activations' type
            return super().emit(emitter)
        emitter.records.append(rec)

    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        from .. import ops
        from ..runtime.program import part_program
        rec = self.record()
        if rec is not None:
            out = torch.empty((x.shape[0], self.H), dtype=torch.float32, device=x.device) if self.out32 else None
            return part_program(self.dtype, x.device, self.H).run_part(rec, x, ctx, out=out)
        if self.activation == "clamped":
            raise ConfigError("gated_mlp: the clamped gate with matrices kept in another element type than the activations")
        gu = self.gate_up(x, out_dtype=torch.float32)[:, :2 * self.ff]
        y = self.down(ops.gated_act(gu, self.bg, self.bu, self.activation, self.dtype), out_dtype=torch.float32)
        if self.bd is not None:
            y = y + self.bd.to(torch.float32)
        return y if self.out32 else y.to(self.dtype)


register_feed_forward("gated_mlp", GatedMLP)
