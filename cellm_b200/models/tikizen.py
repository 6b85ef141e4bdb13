"""Tikizen as a plan: a decoder whose norms sit behind the sums, x <- norm1(alpha x + mixer(x)), x <- norm2(alpha x + ff(x)), so
that the sublayers read the 32-bit stream itself; the embedding's row is normed before the first layer.

Mixers, in the order the configuration lists them:

* `retention`: linear attention with a constant decay per head; turned queries and keys, a norm without weight over a head's
  read-out, a silu gate.
* `attention`: turned (frequencies possibly stretched by their place, YaRN) and then normed queries and keys, inside chunks of
  positions. A layer may read an earlier layer's keys and values: its item of the run order then names that layer's as the
  one whose cache it reads, and the pages there keep what the widest of the readers' masks needs.
* `mamba2`: state-space duality with a short convolution; gate before a norm in groups.

Feed-forwards: the clamped gate (slope 1.702), or routed gated experts (softmax over the chosen) beside a shared expert
behind a sigmoid.

Tensor names: `embed`, `embed.norm`, `final.norm`, `head`, and for layer i `l<i>.norm1|norm2`, `l<i>.mix.q|k|v|g|o` (retention),
`l<i>.mix.q|k|v|o` (attention), `l<i>.mix.in|conv|conv.b|dt_bias|A_log|D|norm|o` (mamba2), `l<i>.mlp.gate|up|down`, or
`l<i>.mlp.router|router.b|e<n>.gate|e<n>.up|e<n>.down|shared.gate|shared.up|shared.down|shared.sg`."""
from __future__ import annotations

from ..config.plan import LayerSpec, ModelPlan, OrderEntry, PartSpec
from ..config.registry import register_architecture
from ..config.tikizen import ChunkedAttention, ClampedMlp, Mamba2, Retention, TikizenConfig

MAX_POSITIONS = 1 << 20      # the design has no limit of its own; angles are formed from 32-bit positions
GATE_SLOPE = 1.702           # of the clamped gate's sigmoid


def _norm(cfg: TikizenConfig, tensor: str) -> PartSpec:
    return PartSpec("rms_norm", {"dim": cfg.width, "eps": cfg.norm_eps}, {"weight": tensor})


def _rope(width: int, rot) -> PartSpec | None:
    if rot is None:
        return None
    return PartSpec("rope", {"head_dim": width, "rotary_dim": rot.dims, "theta": rot.base, "layout": "half",
                             "scaling": rot.scaling.to_dict() if rot.scaling is not None else None})


def kept_keys(cfg: TikizenConfig, j: int) -> dict:
    """What the pages of attention layer j keep for itself and for the layers that read its keys: one chunk's run of positions
    when all of them read chunks of one size, a window of the longest otherwise (a window of c keys holds every chunk of c
    or fewer), everything when one of them reads every earlier key."""
    sizes = {l.mixer.chunk for i, l in enumerate(cfg.layers) if l.type == "attention" and (i == j or l.mixer.kv_from == j)}
    if 0 in sizes:
        return {"kept_chunk": 0}
    return {"kept_chunk": sizes.pop()} if len(sizes) == 1 else {"kept_chunk": 0, "kept_window": max(sizes)}


def _mixer(cfg: TikizenConfig, i: int, p: str) -> PartSpec:
    H, m = cfg.width, cfg.layers[i].mixer
    if isinstance(m, Retention):
        return PartSpec("retention", {"hidden_size": H, "heads": m.heads, "dim": m.dim, "value_dim": m.vdim, "decay": list(m.decay),
                                      "eps": cfg.norm_eps, "position": _rope(m.dim, m.rot), "out_dtype32": True},
                        {k: p + k for k in ("q", "k", "v", "g", "o")})
    if isinstance(m, Mamba2):
        names = {k: p + k for k in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")}
        names["conv_bias"] = p + "conv.b"
        return PartSpec("mamba2", {"hidden_size": H, "heads": m.heads, "value_dim": m.vdim, "state": m.state, "groups": m.groups,
                                   "norm_groups": m.norm_groups, "conv_taps": m.conv, "eps": cfg.norm_eps, "out_dtype32": True}, names)
    assert isinstance(m, ChunkedAttention)
    names = {"q_proj": p + "q", "out_proj": p + "o"}
    if m.kv_from is None:
        names.update(k_proj=p + "k", v_proj=p + "v")
    params = {"hidden_size": H, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "scale": m.scale,
              "chunk": m.chunk, "unit_eps": cfg.norm_eps, "position": _rope(m.dim, m.rot), "reads": m.kv_from is not None, "out_dtype32": True}
    params.update(kept_keys(cfg, i if m.kv_from is None else m.kv_from))
    return PartSpec("turned_attention", params, names)


def _feed_forward(cfg: TikizenConfig, mlp, p: str) -> PartSpec | None:
    if mlp is None:
        return None
    if isinstance(mlp, ClampedMlp):
        return PartSpec("gated_mlp", {"hidden_size": cfg.width, "ff_dim": mlp.ff, "activation": "clamped", "limit": mlp.limit, "slope": GATE_SLOPE,
                                      "out_dtype32": True}, {k: p + k for k in ("gate", "up", "down")})
    names = {"router": p + "router", "correction": p + "router.b"}
    for e in range(mlp.experts):
        names.update({f"{k}_{e}": f"{p}e{e}.{k}" for k in ("gate", "up", "down")})
    if mlp.shared_ff:
        names.update(shared_gate_proj=p + "shared.gate", shared_up=p + "shared.up", shared_down=p + "shared.down", shared_gate=p + "shared.sg")
    return PartSpec("routed_experts", {"hidden_size": cfg.width, "experts": mlp.experts, "top": mlp.top, "ff_dim": mlp.ff, "activation": "silu",
                                       "scores": "softmax", "gated": True, "correction": True, "shared_ff": mlp.shared_ff, "shared_gate": True,
                                       "out_dtype32": True}, names)


def build_plan(cfg: TikizenConfig) -> ModelPlan:
    layers, order = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        layers.append(LayerSpec(PartSpec("post_norm", {"alpha": cfg.postln_alpha}), _mixer(cfg, i, p + "mix."), _feed_forward(cfg, layer.mlp, p + "mlp."),
                                _norm(cfg, p + "norm1"), _norm(cfg, p + "norm2") if layer.mlp is not None else None))
        order.append(OrderEntry(i, layer.mixer.kv_from if layer.type == "attention" else None))
    embedding = PartSpec("lookup", {"vocab_size": cfg.vocab, "dim": cfg.width, "norm_eps": cfg.norm_eps}, {"weight": "embed", "norm": "embed.norm"})
    return ModelPlan(hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS, embedding=embedding,
                     final_norm=_norm(cfg, "final.norm"), head="head", layers=tuple(layers), order=tuple(order), eos_token_id=cfg.eos_token_id,
                     unread_tensors=tuple(f"l{i}.norm2" for i, l in enumerate(cfg.layers) if l.mlp is None))


register_architecture("Tikizen", TikizenConfig, build_plan, model_types=("tikizen",))
