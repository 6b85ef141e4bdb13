"""Gonozen as a plan: a decoder with a norm before and a norm behind every sublayer, x <- x + norm1b(mixer(norm1(x))),
x <- x + norm2b(ff(norm2(x))), two forms of latent attention in the order the configuration lists them, a mixture of experts
behind each, and logits that a tanh holds between two bounds.

* `latent_attention`: one compressed row and one rotated key part a token are cached (rotate-half pairs, frequencies possibly
  stretched by their place, YaRN, whose factor multiplies cos and sin); every earlier row is visible; a head's output is
  multiplied by the sigmoid of a product over the layer's input.
* `latent_attention_2`: queries through a latent of their own, only the compressed row cached, a sliding window, a learned sink
  per head.

Feed-forward: routed experts with the clamped gate (slope 1.702); the scores are the softmax over all experts, the choice is
made within the groups whose largest scores are largest, the chosen scores are divided by their sum; a shared expert with
sizes and a limit of its own is added.

Tensor names: `embed` (also the output matrix), `final.norm`, and for layer i `l<i>.norm1|norm1b|norm2|norm2b`,
`l<i>.mix.q|dkv|dkv.norm|uk|uv|g|o` (latent_attention), `l<i>.mix.dq|dq.norm|uq|dkv|dkv.norm|uk|uv|sink|o` (latent_attention_2),
`l<i>.mlp.router|e<n>.gate|e<n>.up|e<n>.down|shared.gate|shared.up|shared.down`."""
from __future__ import annotations

from ..config.gonozen import GonozenConfig, LatentAttention, Mixture, WindowedLatentAttention
from ..config.plan import LayerSpec, ModelPlan, OrderEntry, PartSpec
from ..config.registry import register_architecture

MAX_POSITIONS = 1 << 20      # the design has no limit of its own; angles are formed from 32-bit positions
GATE_SLOPE = 1.702           # of the clamped gate's sigmoid


def _norm(cfg: GonozenConfig, tensor: str) -> PartSpec:
    return PartSpec("rms_norm", {"dim": cfg.width, "eps": cfg.norm_eps}, {"weight": tensor})


def _mixer(cfg: GonozenConfig, m, p: str) -> PartSpec:
    params = {"hidden_size": cfg.width, "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps}
    names = {"dkv": p + "dkv", "dkv_norm": p + "dkv.norm", "uk": p + "uk", "uv": p + "uv", "o": p + "o"}
    if isinstance(m, LatentAttention):
        rope = None if m.rot is None else PartSpec(
            "rope", {"head_dim": m.rot_dim, "rotary_dim": m.rot.dims, "theta": m.rot.base, "layout": "half",
                     "scaling": m.rot.scaling.to_dict() if m.rot.scaling is not None else None})
        return PartSpec("latent_attention", {**params, "rot_dim": m.rot_dim, "position": rope, "gate": True}, {**names, "q": p + "q", "g": p + "g"})
    assert isinstance(m, WindowedLatentAttention)
    return PartSpec("latent_attention", {**params, "rot_dim": 0, "q_rank": m.q_rank, "window": m.window, "sinks": True},
                    {**names, "dq": p + "dq", "dq_norm": p + "dq.norm", "uq": p + "uq", "sinks": p + "sink"})


def _feed_forward(cfg: GonozenConfig, m: Mixture, p: str) -> PartSpec:
    names = {"router": p + "router"}
    for e in range(m.experts):
        names.update({f"{k}_{e}": f"{p}e{e}.{k}" for k in ("gate", "up", "down")})
    params = {"hidden_size": cfg.width, "experts": m.experts, "top": m.top, "ff_dim": m.expert.ff, "groups": m.groups, "keep_groups": m.keep,
              "scores": "softmax_all", "correction": False, "gated": True, "activation": "clamped", "slope": GATE_SLOPE, "limit": m.expert.limit}
    if m.shared is not None:
        params.update(shared_ff=m.shared.ff, shared_gate=False, shared_limit=m.shared.limit)
        names.update(shared_gate_proj=p + "shared.gate", shared_up=p + "shared.up", shared_down=p + "shared.down")
    return PartSpec("routed_experts", params, names)


def build_plan(cfg: GonozenConfig) -> ModelPlan:
    layers, unread = [], []
    for i, layer in enumerate(cfg.layers):
        p, has_ff = f"l{i}.", layer.mlp is not None
        behind = {"mixer_result_norm": p + "norm1b"}
        if has_ff:
            behind["feed_forward_result_norm"] = p + "norm2b"
        else:
            unread += [p + "norm2", p + "norm2b"]
        block = PartSpec("sandwich_norm", {"hidden_size": cfg.width, "eps": cfg.norm_eps, "feed_forward": has_ff}, behind)
        layers.append(LayerSpec(block, _mixer(cfg, layer.mixer, p + "mix."), _feed_forward(cfg, layer.mlp, p + "mlp.") if has_ff else None,
                                _norm(cfg, p + "norm1"), _norm(cfg, p + "norm2") if has_ff else None))
    head = PartSpec("linear", {"vocab_size": cfg.vocab, "dim": cfg.width, "soft_cap": cfg.logit_softcap}, {"weight": "embed"})
    return ModelPlan(hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS, embedding="embed", final_norm=_norm(cfg, "final.norm"),
                     head=head, layers=tuple(layers), order=tuple(OrderEntry(i) for i in range(len(layers))), eos_token_id=cfg.eos_token_id,
                     unread_tensors=tuple(unread))


register_architecture("Gonozen", GonozenConfig, build_plan, model_types=("gonozen",))
