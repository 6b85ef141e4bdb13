"""A routed feed-forward: many small experts, of which every token runs a few, and optionally one shared expert
that every token runs.

    z = R h (32-bit);  s = sigmoid(z);  c = s + correction
    the experts lie in `groups` equal runs of neighbours; a run's score is the sum of its two largest c; only
    experts of the `keep_groups` best runs can be chosen
    the `top` experts with the largest c are chosen; weight_k = s_k / (sum of the chosen s + 1e-20) * route_scale
    out = sum_k weight_k * D_k act(U_k h)  +  sigmoid(g . h) * D_s act(U_s h)

Two choices are parameters. `scores` "softmax": the `top` experts with the largest z + bias are chosen and weighed by the
softmax over the chosen sums (no sigmoid, no groups); "softmax_all": s is the softmax over all experts, a run's score its
largest, the weights as above. `gated`: an expert (the shared one too) is D (silu(G h) * (U h)), or with the activation
"clamped" D (g' sigmoid(slope g') (u' + 1)) with g' = min(G h, limit), u' = clamp(U h, -limit, limit) (the shared expert has
a limit of its own).

The experts' matrices are kept one below the other, so that a kernel reaches expert e by an offset; gate and up rows of
gated experts lie in blocks of 64, so that the grouped product's epilogue joins the two (widths are padded to multiples of
64 with zeros). The router's rows and the shared expert's gate row form one matrix."""
from __future__ import annotations

import torch

from ..config.errors import ConfigError
from .base import FeedForward, StepContext, TensorSpec
from .gated_mlp import blocked_gate_up, widened_columns
from .linear import stack_rows
from .registry import register_feed_forward

ACTIVATIONS = {"gelu": 0, "gelu_tanh": 1, "silu": 2, "relu": 3}


class RoutedExperts(FeedForward):
    graph_safe = True

    """params: hidden_size, experts, top, ff_dim, activation ("gelu": the exact form), route_scale, groups (default 1),
    keep_groups (default groups), correction (default True), shared_ff (default 0: no shared expert), shared_gate
    (default True), scores ("sigmoid", the default, "softmax" or "softmax_all"), limit, shared_limit (default none) and slope
    (default 1) for gated experts with the activation "clamped", gated (default False), out_dtype32 (default False; gated
    experts only). weights: router [experts, H], correction [experts] (the router's bias under "softmax"), up_<e> [ff, H] and
    down_<e> [H, ff] for every expert e, shared_up [shared_ff, H], shared_down [H, shared_ff], shared_gate [1, H]; and, if
    gated, gate_<e> [ff, H], shared_gate_proj [shared_ff, H]."""

    @classmethod
    def weight_specs(cls, params):
        H, E, ff = params["hidden_size"], params["experts"], params["ff_dim"]
        specs = {"router": TensorSpec((E, H), "linear")}
        if params.get("correction", True):
            specs["correction"] = TensorSpec((E,), "bias")
        for e in range(E):
            if params.get("gated"):
                specs[f"gate_{e}"] = TensorSpec((ff, H), "linear")
            specs[f"up_{e}"] = TensorSpec((ff, H), "linear")
            specs[f"down_{e}"] = TensorSpec((H, ff), "linear")
        sff = params.get("shared_ff", 0)
        if sff:
            if params.get("gated"):
                specs["shared_gate_proj"] = TensorSpec((sff, H), "linear")
            specs["shared_up"] = TensorSpec((sff, H), "linear")
            specs["shared_down"] = TensorSpec((H, sff), "linear")
            if params.get("shared_gate", True):
                specs["shared_gate"] = TensorSpec((1, H), "linear")
        return specs

    def __init__(self, params: dict, weights: dict, dtype: torch.dtype):
        self.H, self.E, self.top, self.ff = (int(params[k]) for k in ("hidden_size", "experts", "top", "ff_dim"))
        self.dtype = dtype
        self.groups = int(params.get("groups", 1))
        self.keep = int(params.get("keep_groups", self.groups))
        self.route_scale = float(params.get("route_scale", 1.0))
        self.activation = params.get("activation", "gelu")
        self.clamped = self.activation == "clamped"
        if self.activation not in ACTIVATIONS and not self.clamped:
            raise ConfigError(f"routed_experts: activation {self.activation!r}; known: {sorted(ACTIVATIONS) + ['clamped']}")
        if self.clamped and not params.get("gated"):
            raise ConfigError("routed_experts: the clamped gate belongs to gated experts")
        none_is_inf = lambda v: float("inf") if v is None else float(v)
        self.limit, self.shared_limit = none_is_inf(params.get("limit")), none_is_inf(params.get("shared_limit"))
        self.slope = float(params.get("slope", 1.0))
        if not 1 <= self.top <= self.E:
            raise ConfigError(f"routed_experts: top {self.top} of {self.E} experts")
        if self.groups < 1 or self.E % self.groups or not 1 <= self.keep <= self.groups:
            raise ConfigError(f"routed_experts: {self.E} experts in {self.groups} groups of which {self.keep} are kept")
        if self.keep * (self.E // self.groups) < self.top:
            raise ConfigError(f"routed_experts: {self.keep} groups of {self.E // self.groups} experts cannot give {self.top} choices")
        self.gated, self.out32 = bool(params.get("gated")), bool(params.get("out_dtype32", False))
        scores = params.get("scores", "sigmoid")
        if scores not in ("sigmoid", "softmax", "softmax_all"):
            raise ConfigError(f"routed_experts: scores {scores!r}; known: 'sigmoid', 'softmax', 'softmax_all'")
        self.softmax = ("sigmoid", "softmax", "softmax_all").index(scores)
        if self.softmax == 1 and self.groups != 1:
            raise ConfigError("routed_experts: groups of experts under softmax scores are not built")
        if self.out32 and not self.gated:
            raise ConfigError("routed_experts: a 32-bit result is built for gated experts")
        if self.gated:
            self.up = stack_rows(*[blocked_gate_up(weights[f"gate_{e}"], weights[f"up_{e}"]) for e in range(self.E)])
            self.down = stack_rows(*[widened_columns(weights[f"down_{e}"]) for e in range(self.E)])
            self.ff = int(self.down.shape[1])
        else:
            self.up = stack_rows(*[weights[f"up_{e}"] for e in range(self.E)])
            self.down = stack_rows(*[weights[f"down_{e}"] for e in range(self.E)])
        dev = self.up.device
        self.shared_ff = int(params.get("shared_ff", 0))
        self.has_gate = bool(self.shared_ff and params.get("shared_gate", True))
        self.router = stack_rows(weights["router"], weights["shared_gate"]) if self.has_gate else weights["router"].contiguous()
        self.correction = (weights["correction"].contiguous() if params.get("correction", True)
                           else torch.zeros(self.E, dtype=torch.float32, device=dev))
        if self.gated and self.shared_ff:
            self.shared_up = blocked_gate_up(weights["shared_gate_proj"], weights["shared_up"])
            self.shared_down = widened_columns(weights["shared_down"])
            self.shared_ff = int(self.shared_down.shape[1])
        else:
            self.shared_up = weights["shared_up"].contiguous() if self.shared_ff else None
            self.shared_down = weights["shared_down"].contiguous() if self.shared_ff else None
        self._record = None

    def record(self):
        from ..ops._lib import tag
        from ..runtime import records as R
        mats = [self.up, self.down, self.router] + ([self.shared_up, self.shared_down] if self.shared_ff else [])
        if self._record is None and all(m.dtype == self.dtype for m in mats):
            p = R.RoutedMlpParams()
            p.up, p.down, p.router = R.linear(self.up), R.linear(self.down), R.linear(self.router)
            p.correction, p.c_dtype = self.correction.data_ptr(), tag(self.correction)
            p.experts, p.top, p.n_groups, p.keep, p.scale = self.E, self.top, self.groups, self.keep, self.route_scale
            p.ff, p.act = self.ff, ACTIVATIONS.get(self.activation, 0)
            p.gate_kind, p.limit, p.shared_limit, p.slope = int(self.clamped), self.limit, self.shared_limit, self.slope
            if self.shared_ff:
                p.shared_up, p.shared_down = R.linear(self.shared_up), R.linear(self.shared_down)
            p.shared_ff, p.shared_gate = self.shared_ff, int(self.has_gate)
            p.gated, p.softmax, p.out32 = int(self.gated), int(self.softmax), int(self.out32)
            self._record = R.Record(R.ROUTED_MLP, p, part=self)
        return self._record

    def emit(self, emitter) -> None:
        rec = self.record()
        if rec is None:
            raise ConfigError("routed_experts: matrices kept in another element type than the activations")
        if self.out32:                      # the executor's registers hold results in the activations' type
            return super().emit(emitter)
        emitter.records.append(rec)

    def forward(self, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        from ..runtime.program import part_program
        rec = self.record()
        if rec is None:
            raise ConfigError("routed_experts: matrices kept in another element type than the activations")
        out = torch.empty((x.shape[0], self.H), dtype=torch.float32, device=x.device) if self.out32 else None
        return part_program(self.dtype, x.device, self.H).run_part(rec, x, ctx, out=out)


register_feed_forward("routed_experts", RoutedExperts)
