"""``RupenexConfig``: the keys of a Rupenex ``config.json`` as the engine reads them.

    architecture   "Rupenex"
    vocab, width   sizes of the embedding
    norm           {eps}: of every norm of the model
    logit_scale    the logits are multiplied by it (absent: 1)
    layers         a list; each entry {type, mixer, mlp}:
                   type "attention": mixer {heads, kv_heads, dim, vdim, scale, mask {size, keep_first},
                       rot {base, dims, scaling {factor}}}
                       a window of mask.size keys beside the first mask.keep_first keys of the sequence (mask absent: plain
                       causal; keep_first absent: none); rot absent: no rotation; scaling absent: plain frequencies
                   type "mamba2": mixer {heads, vdim, state, groups, conv, norm_groups}
                       heads values of size vdim, groups pairs of input and output vectors of size state, conv taps,
                       the norm's row in norm_groups parts
                   mlp null | {kind "dense", ff, limit}
                            | {kind "moe", expert {ff}, router {experts, top, identity}, shared {ff}}
                       identity absent: no identity experts; shared absent: no expert that every token runs

Everything a model of this design may vary is read from here; nothing is defaulted to the
values of one particular model.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ConfigError, ModelConfig, take_float, take_int
from .ronurax import _obj


@dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int
    factor: Optional[float]         # every frequency is divided by it; None: plain frequencies

    def to_dict(self):
        d = {"base": self.base, "dims": self.dims}
        if self.factor is not None:
            d["scaling"] = {"factor": self.factor}
        return d


@dataclass(frozen=True)
class SinkAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]           # mask.size; None: plain causal
    keep_first: int                 # first keys of the sequence that stay visible beside the window
    rot: Optional[RotationConfig]

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.window is not None:
            d["mask"] = {"size": self.window}
            if self.keep_first:
                d["mask"]["keep_first"] = self.keep_first
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    def to_dict(self):
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class RupenexMlpConfig:
    kind: str                       # "dense" | "moe"
    ff: int                         # of the dense layer, or of an expert
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    identity: int = 0
    shared_ff: int = 0              # 0: no expert that every token runs

    def to_dict(self):
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff, "limit": self.limit}
        d = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}
        if self.identity:
            d["router"]["identity"] = self.identity
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


@dataclass(frozen=True)
class RupenexLayerConfig:
    type: str                       # "attention" | "mamba2"
    mixer: object
    mlp: Optional[RupenexMlpConfig]

    def to_dict(self):
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp else None}


def _sizes(m, *keys):
    return [take_int(m, k, minimum=1) for k in keys]


def _rotation(m, where, dim):
    r = m.get("rot")
    if r is None:
        return None
    r = _obj(m, "rot", where)
    base, dims = take_float(r, "base"), take_int(r, "dims", minimum=2)
    if dims % 2 or dims > dim or base <= 0:
        raise ConfigError(f"{where}: rot.dims {dims} must be even and within the head's {dim}, rot.base {base} positive")
    factor = None
    if r.get("scaling") is not None:
        factor = take_float(_obj(r, "scaling", where), "factor")
        if not factor > 0:
            raise ConfigError(f"{where}: rot.scaling.factor must be positive, got {factor}")
    return RotationConfig(base, dims, factor)


def _mixer(kind, m, where):
    if kind == "attention":
        heads, kv, dim, vdim = _sizes(m, "heads", "kv_heads", "dim", "vdim")
        if heads % kv:
            raise ConfigError(f"{where}: {heads} heads are not a multiple of {kv} kv_heads")
        window, keep = None, 0
        if m.get("mask") is not None:
            mask = _obj(m, "mask", where)
            window, keep = take_int(mask, "size", minimum=1), take_int(mask, "keep_first", 0, minimum=0)
        return SinkAttentionConfig(heads, kv, dim, vdim, take_float(m, "scale"), window, keep, _rotation(m, where, dim))
    if kind != "mamba2":
        raise ConfigError(f"{where}: unknown layer type {kind!r} (attention, mamba2)")
    c = Mamba2Config(*_sizes(m, "heads", "vdim", "state", "groups", "conv", "norm_groups"))
    if c.heads % c.groups or (c.heads * c.vdim) % c.norm_groups:
        raise ConfigError(f"{where}: {c.heads} heads in {c.groups} groups, {c.heads * c.vdim} channels in {c.norm_groups} "
                          "parts of the norm: both must divide")
    return c


def _mlp(ml, where):
    if ml is None:
        return None
    if not isinstance(ml, dict):
        raise ConfigError(f"{where}: 'mlp' must be an object or null")
    if ml.get("kind") == "dense":
        limit = take_float(ml, "limit")
        if not limit > 0:
            raise ConfigError(f"{where}: mlp.limit must be positive, got {limit}")
        return RupenexMlpConfig("dense", take_int(ml, "ff", minimum=1), limit)
    if ml.get("kind") != "moe":
        raise ConfigError(f"{where}: unknown mlp kind {ml.get('kind')!r} (dense, moe)")
    r = _obj(ml, "router", where)
    experts, top = _sizes(r, "experts", "top")
    identity = take_int(r, "identity", 0, minimum=0)
    if top > experts + identity:
        raise ConfigError(f"{where}: top {top} of {experts} experts and {identity} identity experts")
    shared = take_int(_obj(ml, "shared", where), "ff", minimum=1) if ml.get("shared") is not None else 0
    return RupenexMlpConfig("moe", take_int(_obj(ml, "expert", where), "ff", minimum=1), 0.0, experts, top, identity, shared)


@dataclass(frozen=True)
class RupenexConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    layers: Tuple[RupenexLayerConfig, ...]

    @classmethod
    def from_dict(cls, d: dict) -> "RupenexConfig":
        vocab, width = _sizes(d, "vocab", "width")
        eps = take_float(_obj(d, "norm"), "eps")
        if eps <= 0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {eps}")
        scale = take_float(d, "logit_scale", 1.0)
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw):
            where = f"config.json: layers[{i}]"
            if not isinstance(L, dict):
                raise ConfigError(f"{where} must be an object")
            layers.append(RupenexLayerConfig(L.get("type"), _mixer(L.get("type"), _obj(L, "mixer", where), where),
                                             _mlp(L.get("mlp"), where)))
        return cls(architecture="Rupenex", vocab=vocab, width=width, norm_eps=eps, logit_scale=scale, layers=tuple(layers))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "logit_scale": self.logit_scale, "layers": [L.to_dict() for L in self.layers]}
