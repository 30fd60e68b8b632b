"""``DiraraxConfig``: the keys of a Dirarax ``config.json`` as the engine reads them.

    architecture   "Dirarax"
    vocab, width   sizes of the embedding, which is also the head
    norm           {eps}: of every norm of the model
    layers         a list; each entry {type, mixer, mlp}:
                   type "gla":      mixer {heads, dim, vdim, tau}
                       linear attention with a gated decay per key channel
                   type "parallel": mixer {left, right, left_scale, right_scale}: two mixers side by side
                       left  {heads, kv_heads, dim, vdim, scale, rot {base, dims, scaling {factor, original, fast, slow}}}
                             gated grouped attention; rot absent: no rotation; scaling absent: plain frequencies
                       right {heads, dim, vdim, decay [one number per head], rot {base, dims}}
                             linear attention with a fixed decay per head
                   mlp null | {kind "dense", ff} | {kind "moe", expert {ff}, router {experts, top}, shared {ff}}
                       shared absent: no expert that every token runs
    loop           {start, stop, times} (optional): layers start .. stop-1 run ``times`` times in a row; a mix with the
                   embedding's output and a vector of its own stand before every pass

Everything a model of this design may vary is read from here; nothing is defaulted to the
values of one particular model.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ConfigError, ModelConfig, take_float, take_int
from .ronurax import RotaryConfig, _obj, _rotary


@dataclass(frozen=True)
class GatedLinearConfig:
    heads: int
    dim: int
    vdim: int
    tau: float

    def to_dict(self):
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "tau": self.tau}


@dataclass(frozen=True)
class GatedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotaryConfig]

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Optional[RotaryConfig]

    def to_dict(self):
        d = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class ParallelConfig:
    left: GatedAttentionConfig
    right: RetentionConfig
    left_scale: float
    right_scale: float

    def to_dict(self):
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                "right_scale": self.right_scale}


@dataclass(frozen=True)
class MlpConfig:
    kind: str                   # "dense" | "moe"
    ff: int                     # of the dense layer, or of one expert
    experts: int = 0
    top: int = 0
    shared_ff: int = 0          # 0: no expert that every token runs

    def to_dict(self):
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        d = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


@dataclass(frozen=True)
class LayerConfig:
    type: str                   # "gla" | "parallel"
    mixer: object
    mlp: Optional[MlpConfig]

    def to_dict(self):
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp else None}


def _sizes(m, *keys):
    return [take_int(m, k, minimum=1) for k in keys]


def _rot(m, where, dim, keys):
    rot = _rotary(m, where, keys)
    if rot is not None and rot.dims > dim:
        raise ConfigError(f"{where}: rot.dims {rot.dims} beyond the head's {dim}")
    return rot


def _mixer(kind, m, where):
    if kind == "gla":
        tau = take_float(m, "tau")
        if not tau > 0:
            raise ConfigError(f"{where}: tau must be positive, got {tau}")
        return GatedLinearConfig(*_sizes(m, "heads", "dim", "vdim"), tau)
    if kind != "parallel":
        raise ConfigError(f"{where}: unknown layer type {kind!r} (gla, parallel)")
    a, r = _obj(m, "left", where), _obj(m, "right", where)
    heads, kv, dim, vdim = _sizes(a, "heads", "kv_heads", "dim", "vdim")
    if heads % kv:
        raise ConfigError(f"{where}: {heads} heads are not a multiple of {kv} kv_heads")
    left = GatedAttentionConfig(heads, kv, dim, vdim, take_float(a, "scale"),
                                _rot(a, where + ".left", dim, ("factor", "original", "fast", "slow")))
    heads, dim, vdim = _sizes(r, "heads", "dim", "vdim")
    decay = r.get("decay")
    if not isinstance(decay, list) or len(decay) != heads or not all(
            isinstance(v, (int, float)) and not isinstance(v, bool) and 0.0 < v <= 1.0 for v in decay):
        raise ConfigError(f"{where}: 'decay' must list one number in (0, 1] for each of the {heads} heads")
    right = RetentionConfig(heads, dim, vdim, tuple(float(v) for v in decay), _rot(r, where + ".right", dim, ()))
    return ParallelConfig(left, right, take_float(m, "left_scale"), take_float(m, "right_scale"))


def _mlp(ml, where):
    if ml is None:
        return None
    if not isinstance(ml, dict):
        raise ConfigError(f"{where}: 'mlp' must be an object or null")
    if ml.get("kind") == "dense":
        return MlpConfig("dense", take_int(ml, "ff", minimum=1))
    if ml.get("kind") != "moe":
        raise ConfigError(f"{where}: unknown mlp kind {ml.get('kind')!r} (dense, moe)")
    r = _obj(ml, "router", where)
    experts, top = _sizes(r, "experts", "top")
    if top > experts:
        raise ConfigError(f"{where}: top {top} of {experts} experts")
    shared = take_int(_obj(ml, "shared", where), "ff", minimum=1) if ml.get("shared") is not None else 0
    return MlpConfig("moe", take_int(_obj(ml, "expert", where), "ff", minimum=1), experts, top, shared)


@dataclass(frozen=True)
class DiraraxConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[LayerConfig, ...]
    loop_start: int
    loop_stop: int
    loop_times: int             # 0: no loop

    @classmethod
    def from_dict(cls, d: dict) -> "DiraraxConfig":
        vocab, width = _sizes(d, "vocab", "width")
        eps = take_float(_obj(d, "norm"), "eps")
        if eps <= 0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {eps}")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw):
            where = f"config.json: layers[{i}]"
            if not isinstance(L, dict):
                raise ConfigError(f"{where} must be an object")
            layers.append(LayerConfig(L.get("type"), _mixer(L.get("type"), _obj(L, "mixer", where), where),
                                      _mlp(L.get("mlp"), where)))
        loop, start, stop, times = d.get("loop"), 0, 0, 0
        if loop is not None:
            if not isinstance(loop, dict):
                raise ConfigError("config.json: 'loop' must be an object")
            start, stop = take_int(loop, "start", minimum=0), take_int(loop, "stop", minimum=0)
            times = take_int(loop, "times", minimum=1)
            if not (start < stop <= len(layers)):
                raise ConfigError(f"config.json: loop {start}..{stop} does not lie within the {len(layers)} layers")
        return cls(architecture="Dirarax", vocab=vocab, width=width, norm_eps=eps, layers=tuple(layers), loop_start=start,
                   loop_stop=stop, loop_times=times)

    def layer_order(self):
        """[(layer, pass or None)] in the order they run; a pass number stands at the first layer of each pass."""
        n, a, b = len(self.layers), self.loop_start, self.loop_stop
        if not self.loop_times:
            return [(i, None) for i in range(n)]
        passes = [(i, t if i == a else None) for t in range(self.loop_times) for i in range(a, b)]
        return [(i, None) for i in range(a)] + passes + [(i, None) for i in range(b, n)]

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": [L.to_dict() for L in self.layers]}
        if self.loop_times:
            d["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        return d
