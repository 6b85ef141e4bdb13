"""Typed configuration of the Gonozen design, read from its config.json.

The file names the design with one string (`architecture`) and gives the vocabulary, the model's width, the norms' eps, the
bound of the logits (`logit_softcap`) and the list of layers. A layer has a `type` (its mixer), the mixer's sizes and
constants (`mixer`) and its feed-forward (`mlp`, or null for none).

Mixer types: `latent_attention` (a rotated key part beside the latent, a gate per head on the output) and
`latent_attention_2` (queries through a latent of their own, no rotation, a sliding window, a sink per head). The one
feed-forward kind is `moe` (routed experts with the clamped gate, chosen within groups). Every size and constant that can
differ between models comes from the file; what the file leaves out does not exist (no `mask`: every earlier row; no `rot`
or no `scaling`: no rotation or plain frequencies; no `limit`: no clamping; no `groups`: one group; no `shared`: no shared
expert; no `logit_softcap`: logits as they are)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .errors import ConfigError
from .lfm2 import _get
from .padadra import _obj
from .tikizen import Rot, _rot

MIXERS = ("latent_attention", "latent_attention_2")
MLP_KINDS = ("moe",)


def _positive(where: str, *sizes: int) -> None:
    if min(sizes) < 1:
        raise ConfigError(f"config.json: {where}: sizes must be positive")


@dataclass(frozen=True)
class LatentAttention:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Optional[Rot]

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "LatentAttention":
        sizes = [_get(d, k, int) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")]
        c = cls(*sizes, _get(d, "scale", float), _rot(d, where, sizes[2]))
        _positive(where, c.heads, c.dim, c.vdim, c.kv_rank)
        if c.rot_dim < 0:
            raise ConfigError(f"config.json: {where}: rot_dim must not be negative")
        return c

    def to_dict(self) -> dict:
        d = {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "rot_dim": self.rot_dim, "scale": self.scale, "vdim": self.vdim}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class WindowedLatentAttention:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    window: int                 # 0: every earlier row

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "WindowedLatentAttention":
        mask = _obj(d, "mask", where, required=False)
        window = _get(mask, "size", int) if mask is not None else 0
        c = cls(*(_get(d, k, int) for k in ("heads", "dim", "vdim", "kv_rank", "q_rank")), _get(d, "scale", float), window)
        _positive(where, c.heads, c.dim, c.vdim, c.kv_rank, c.q_rank)
        if mask is not None and window < 1:
            raise ConfigError(f"config.json: {where}.mask.size must be positive")
        return c

    def to_dict(self) -> dict:
        d = {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "q_rank": self.q_rank, "scale": self.scale, "vdim": self.vdim}
        if self.window:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class ClampedExpert:
    ff: int
    limit: Optional[float]

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "ClampedExpert":
        c = cls(_get(d, "ff", int), _get(d, "limit", float, None))
        _positive(where, c.ff)
        return c

    def to_dict(self) -> dict:
        return {"ff": self.ff} if self.limit is None else {"ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class Mixture:
    expert: ClampedExpert
    shared: Optional[ClampedExpert]
    experts: int
    top: int
    groups: int
    keep: int

    @classmethod
    def from_dict(cls, d, where: str) -> Optional["Mixture"]:
        if d is None:
            return None
        if not isinstance(d, dict):
            raise ConfigError(f"config.json: {where} should be an object or null")
        kind = _get(d, "kind", str)
        if kind not in MLP_KINDS:
            raise ConfigError(f"config.json: {where}: feed-forward kind {kind!r}; known: {list(MLP_KINDS)}")
        router, shared = _obj(d, "router", where), _obj(d, "shared", where, required=False)
        groups = _obj(router, "groups", where + ".router", required=False)
        count = _get(groups, "count", int) if groups is not None else 1
        c = cls(ClampedExpert.from_dict(_obj(d, "expert", where), where + ".expert"),
                ClampedExpert.from_dict(shared, where + ".shared") if shared is not None else None,
                _get(router, "experts", int), _get(router, "top", int), count, _get(groups, "keep", int) if groups is not None else 1)
        if not 1 <= c.top <= c.experts:
            raise ConfigError(f"config.json: {where}.router: top {c.top} of {c.experts} experts")
        if c.groups < 1 or c.experts % c.groups or not 1 <= c.keep <= c.groups or c.keep * (c.experts // c.groups) < c.top:
            raise ConfigError(f"config.json: {where}.router.groups: {c.experts} experts in {c.groups} groups of which {c.keep} are kept cannot "
                              f"give {c.top} choices")
        return c

    def to_dict(self) -> dict:
        router = {"experts": self.experts, "top": self.top}
        if self.groups > 1:
            router["groups"] = {"count": self.groups, "keep": self.keep}
        d = {"expert": self.expert.to_dict(), "kind": "moe", "router": router}
        if self.shared is not None:
            d["shared"] = self.shared.to_dict()
        return d


@dataclass(frozen=True)
class GonozenLayer:
    type: str
    mixer: object               # LatentAttention | WindowedLatentAttention
    mlp: Optional[Mixture]

    def to_dict(self) -> dict:
        return {"mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None, "type": self.type}


@dataclass(frozen=True)
class GonozenConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_softcap: Optional[float]
    layers: tuple
    eos_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict) -> "GonozenConfig":
        readers = {"latent_attention": LatentAttention, "latent_attention_2": WindowedLatentAttention}
        layers = []
        for i, entry in enumerate(_get(d, "layers", list)):
            where = f"layers[{i}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"config.json: {where} should be an object")
            kind = _get(entry, "type", str)
            if kind not in readers:
                raise ConfigError(f"config.json: {where}: mixer type {kind!r}; known: {list(MIXERS)}")
            layers.append(GonozenLayer(kind, readers[kind].from_dict(_get(entry, "mixer", dict), where + ".mixer"),
                                       Mixture.from_dict(entry.get("mlp"), where + ".mlp")))
        c = cls(_get(d, "vocab", int), _get(d, "width", int), _get(_get(d, "norm", dict), "eps", float), _get(d, "logit_softcap", float, None),
                tuple(layers), _get(d, "eos_token_id", int, None))
        if c.vocab < 1 or c.width < 1:
            raise ConfigError("config.json: vocab and width must be positive")
        if c.logit_softcap is not None and not c.logit_softcap > 0:
            raise ConfigError("config.json: logit_softcap must be positive")
        return c

    def to_dict(self) -> dict:
        d = {"architecture": "Gonozen", "layers": [l.to_dict() for l in self.layers], "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
             "width": self.width}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d
