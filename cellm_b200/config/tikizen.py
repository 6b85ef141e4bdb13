"""Typed configuration of the Tikizen design, read from its config.json.

The file names the design with one string (`architecture`) and gives the vocabulary, the model's width, the norms' eps, the
factor of the stream in every sum before a norm (`postln_alpha`) and the list of layers. A layer has a `type` (its mixer),
the mixer's sizes and constants (`mixer`) and its feed-forward (`mlp`, or null for none).

Mixer types: `retention` (linear attention with a constant decay per head), `attention` (turned and normed queries and keys
inside chunks of positions; it may name an earlier layer whose keys and values it reads, `kv_from`) and `mamba2` (state-space
duality). Feed-forward kinds: `dense` (the clamped gate) and `moe` (routed gated experts beside a shared one). Every size
and constant that can differ between models comes from the file; what the file leaves out does not exist (no `mask`: every
earlier key; no `rot`: no rotation; no `scaling`: plain frequencies; no `limit`: no clamping; no `shared`: no shared expert)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .errors import ConfigError
from .lfm2 import _get
from .padadra import _obj

MIXERS = ("retention", "attention", "mamba2")
MLP_KINDS = ("dense", "moe")


@dataclass(frozen=True)
class PlaceScaling:
    factor: float
    original: float
    fast: float
    slow: float

    def to_dict(self) -> dict:
        return {"factor": self.factor, "fast": self.fast, "original": self.original, "slow": self.slow}


@dataclass(frozen=True)
class Rot:
    base: float
    dims: int
    scaling: Optional[PlaceScaling]

    def to_dict(self) -> dict:
        d = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = self.scaling.to_dict()
        return d


def _rot(d: dict, where: str, limit: int) -> Optional[Rot]:
    r = _obj(d, "rot", where, required=False)
    if r is None:
        return None
    sc = _obj(r, "scaling", where + ".rot", required=False)
    if sc is not None:
        sc = PlaceScaling(*(_get(sc, k, float) for k in ("factor", "original", "fast", "slow")))
        if min(sc.factor, sc.original, sc.fast, sc.slow) <= 0:
            raise ConfigError(f"config.json: {where}.rot.scaling needs positive numbers")
    rot = Rot(_get(r, "base", float), _get(r, "dims", int), sc)
    if rot.dims % 2 or not 0 <= rot.dims <= limit or rot.base <= 0:
        raise ConfigError(f"config.json: {where}.rot: dims must be even and at most {limit}, base positive")
    return rot if rot.dims else None


@dataclass(frozen=True)
class Retention:
    heads: int
    dim: int
    vdim: int
    decay: tuple
    rot: Optional[Rot]

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "Retention":
        heads, dim = _get(d, "heads", int), _get(d, "dim", int)
        decay = _get(d, "decay", list)
        if any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in decay):
            raise ConfigError(f"config.json: {where}.decay should be a list of numbers")
        c = cls(heads, dim, _get(d, "vdim", int, dim), tuple(float(x) for x in decay), _rot(d, where, dim))
        if min(c.heads, c.dim, c.vdim) < 1:
            raise ConfigError(f"config.json: {where}: sizes must be positive")
        if len(c.decay) != c.heads:
            raise ConfigError(f"config.json: {where}: {len(c.decay)} numbers in decay for {c.heads} heads")
        return c

    def to_dict(self) -> dict:
        d = {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class ChunkedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int                  # 0: every earlier key
    kv_from: Optional[int]      # the layer whose keys and values it reads
    rot: Optional[Rot]

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "ChunkedAttention":
        heads, dim = _get(d, "heads", int), _get(d, "dim", int)
        mask = _obj(d, "mask", where, required=False) or {}
        c = cls(heads, _get(d, "kv_heads", int, heads), dim, _get(d, "vdim", int, dim), _get(d, "scale", float), _get(mask, "size", int, 0),
                _get(d, "kv_from", int, None), _rot(d, where, dim))
        if min(c.heads, c.kv_heads, c.dim, c.vdim) < 1 or c.chunk < 0:
            raise ConfigError(f"config.json: {where}: sizes must be positive")
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}: {c.heads} heads are not a multiple of {c.kv_heads} key/value heads")
        return c

    def to_dict(self) -> dict:
        d = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.chunk:
            d["mask"] = {"size": self.chunk}
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class Mamba2:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "Mamba2":
        c = cls(_get(d, "heads", int), _get(d, "vdim", int), _get(d, "state", int), _get(d, "groups", int, 1), _get(d, "norm_groups", int, 1),
                _get(d, "conv", int))
        if min(c.heads, c.vdim, c.state, c.groups, c.norm_groups, c.conv) < 1:
            raise ConfigError(f"config.json: {where}: sizes must be positive")
        if c.heads % c.groups:
            raise ConfigError(f"config.json: {where}: {c.heads} heads are not a multiple of {c.groups} groups")
        if (c.heads * c.vdim) % c.norm_groups:
            raise ConfigError(f"config.json: {where}: {c.heads * c.vdim} values do not form {c.norm_groups} equal parts (norm_groups)")
        return c

    def to_dict(self) -> dict:
        return {"conv": self.conv, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups, "state": self.state, "vdim": self.vdim}


@dataclass(frozen=True)
class ClampedMlp:
    ff: int
    limit: Optional[float]

    def to_dict(self) -> dict:
        d = {"ff": self.ff, "kind": "dense"}
        if self.limit is not None:
            d["limit"] = self.limit
        return d


@dataclass(frozen=True)
class Mixture:
    ff: int
    experts: int
    top: int
    shared_ff: int          # 0: no shared expert

    def to_dict(self) -> dict:
        d = {"expert": {"ff": self.ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


def _mlp(d, where: str):
    if d is None:
        return None
    if not isinstance(d, dict):
        raise ConfigError(f"config.json: {where} should be an object or null")
    kind = _get(d, "kind", str)
    if kind not in MLP_KINDS:
        raise ConfigError(f"config.json: {where}: feed-forward kind {kind!r}; known: {list(MLP_KINDS)}")
    if kind == "dense":
        c = ClampedMlp(_get(d, "ff", int), _get(d, "limit", float, None))
        if c.ff < 1:
            raise ConfigError(f"config.json: {where}: ff must be positive")
        return c
    router, expert = _obj(d, "router", where), _obj(d, "expert", where)
    shared = _obj(d, "shared", where, required=False)
    c = Mixture(_get(expert, "ff", int), _get(router, "experts", int), _get(router, "top", int), _get(shared, "ff", int) if shared is not None else 0)
    if c.ff < 1 or c.shared_ff < 0 or not 1 <= c.top <= c.experts:
        raise ConfigError(f"config.json: {where}: expert sizes must be positive and top at most the number of experts")
    return c


@dataclass(frozen=True)
class TikizenLayer:
    type: str
    mixer: object           # Retention | ChunkedAttention | Mamba2
    mlp: object             # ClampedMlp | Mixture | None

    def to_dict(self) -> dict:
        return {"mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp is not None else None, "type": self.type}


@dataclass(frozen=True)
class TikizenConfig:
    vocab: int
    width: int
    norm_eps: float
    postln_alpha: float
    layers: tuple
    eos_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict) -> "TikizenConfig":
        norm = _get(d, "norm", dict)
        readers = {"retention": Retention, "attention": ChunkedAttention, "mamba2": Mamba2}
        layers = []
        for i, entry in enumerate(_get(d, "layers", list)):
            where = f"layers[{i}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"config.json: {where} should be an object")
            kind = _get(entry, "type", str)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}: mixer type {kind!r}; known: {list(MIXERS)}")
            layers.append(TikizenLayer(kind, readers[kind].from_dict(_get(entry, "mixer", dict), where + ".mixer"), _mlp(entry.get("mlp"), where + ".mlp")))
        for i, layer in enumerate(layers):
            j = layer.mixer.kv_from if layer.type == "attention" else None
            if j is None:
                continue
            if not 0 <= j < i or layers[j].type != "attention" or layers[j].mixer.kv_from is not None:
                raise ConfigError(f"config.json: layers[{i}].mixer.kv_from must name an earlier attention layer with keys and values of its own, not {j}")
            a, b = layer.mixer, layers[j].mixer
            if (a.kv_heads, a.dim, a.vdim) != (b.kv_heads, b.dim, b.vdim):
                raise ConfigError(f"config.json: layers[{i}].mixer.kv_from: the key/value heads of layer {j} are of other sizes")
        c = cls(_get(d, "vocab", int), _get(d, "width", int), _get(norm, "eps", float), _get(d, "postln_alpha", float, 1.0), tuple(layers),
                _get(d, "eos_token_id", int, None))
        if c.vocab < 1 or c.width < 1:
            raise ConfigError("config.json: vocab and width must be positive")
        return c

    def to_dict(self) -> dict:
        d = {"architecture": "Tikizen", "layers": [l.to_dict() for l in self.layers], "norm": {"eps": self.norm_eps},
             "postln_alpha": self.postln_alpha, "vocab": self.vocab, "width": self.width}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d
