"""Descriptions from which a model is assembled, and the registries of part kinds.

An architecture turns its typed configuration into a ``ModelSpec``: plain data that
names, layer by layer, which mixer, feed-forward, norm and block arrangement to
build, with every size and constant as a parameter, and in which order the layers
run.  ``kllm_b200.parts.model.DecoderModel`` builds the parts through the
registries below; no part is told which model it is in.

The order of execution is data too: ``ModelSpec.schedule`` is a list of
``LayerCall(block, cache, writes_cache)``.  A block index may appear twice (the
same weights run again, each call with a cache slot of its own), and a call may
name the cache slot of another call with ``writes_cache=False`` to read keys and
values that an earlier layer wrote.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional, Tuple


@dataclass(frozen=True)
class TensorSpec:
    """One tensor a part expects from the weight files.

    store: "compute" -> kept in the model's dtype (bfloat16 or float32);
           "float32" -> kept in 32-bit whatever the model's dtype (norm gains,
           router tables); "int32" -> integer table.
    init:  how random-weights mode fills it: "normal" (mean 0), "gain" (mean 1),
           "zeros", "uniform:lo:hi", "eye" (the identity), "mean" (1 / first size), or for an
           integer table "distinct:B" (rows of different values below B); the spreads are
           arguments of that mode.
    optional: may be absent from the files (the part then copes, e.g. a tied head).
    free:  indices of dimensions whose size the files decide (a rank that no configuration
           key names); ``shape`` then holds the size that random-weights mode draws, and the
           part reads the real one from the tensor it is bound to.
    """
    name: str
    shape: Tuple[int, ...]
    store: str = "compute"
    init: str = "normal"
    optional: bool = False
    free: Tuple[int, ...] = ()

    def fits(self, shape) -> bool:
        shape = tuple(shape)
        return len(shape) == len(self.shape) and all(
            a == b or (i in self.free and a > 0) for i, (a, b) in enumerate(zip(shape, self.shape)))


@dataclass
class PartSpec:
    kind: str
    prefix: str = ""
    params: Dict = field(default_factory=dict)


@dataclass
class BlockSpec:
    """One layer: an arrangement (``kind``) of a mixer, a feed-forward and norms."""
    kind: str
    prefix: str
    mixer: PartSpec
    feed_forward: Optional[PartSpec]     # None where the arrangement allows a layer without one
    mixer_norm: PartSpec
    ff_norm: Optional[PartSpec]
    params: Dict = field(default_factory=dict)


@dataclass(frozen=True)
class LayerCall:
    block: int
    cache: int
    writes_cache: bool = True
    entry: Optional[Tuple[int, int]] = None     # (index into ModelSpec.entries, its argument): done to the stream before the layer


@dataclass
class ModelSpec:
    hidden_size: int
    vocab_size: int
    max_position: int
    embedding: PartSpec
    blocks: List[BlockSpec]
    schedule: List[LayerCall]
    final_norm: PartSpec
    head: PartSpec
    eos_token_ids: Tuple[int, ...] = ()
    entries: List[PartSpec] = field(default_factory=list)   # parts of the stream_entry family that schedule entries name


# ---- what a mixer asks of the cache manager ---------------------------------

@dataclass(frozen=True)
class PagedKVNeed:
    """Keys and values in pages.  window None: every key is kept; window W: only
    the last W keys of a request are ever read, older pages may be given back.
    keep_first: beside a window, the first so many keys of a request are read as well and their pages stay.
    v_head_dim: the size of a head's values where it differs from the keys' (None: the same).
    values_are_keys: one row per token serves as key and as value (a layer that attends
    through a cached low-rank latent): no value store is kept, the views of the values are the
    keys'; with a ``v_head_dim`` below ``head_dim`` the values are the first ``v_head_dim`` elements
    of that row (a row that carries something beside the latent for the keys alone).
    n_v_heads: the heads of the value store where they are fewer than the key heads (None: the
    same): n_kv_heads / n_v_heads neighbouring key heads attend over one value head."""
    n_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    v_head_dim: Optional[int] = None
    values_are_keys: bool = False
    n_v_heads: Optional[int] = None
    keep_first: int = 0

    @property
    def value_dim(self) -> int:
        return self.v_head_dim or self.head_dim

    @property
    def value_heads(self) -> int:
        return self.n_v_heads or self.n_kv_heads

    @property
    def stored_dim(self) -> int:
        """Elements kept per token and kv head (with the same number of key and value heads)."""
        return self.head_dim if self.values_are_keys else self.head_dim + self.value_dim

    @property
    def stored_per_token(self) -> int:
        """Elements kept per token over all heads."""
        keys = self.n_kv_heads * self.head_dim
        return keys if self.values_are_keys else keys + self.value_heads * self.value_dim


@dataclass(frozen=True)
class StateNeed:
    """Per-request state of fixed size, one slot per live request, zero at the
    start of a request.  A layer that asks for several gives all but one a ``name``
    (``LayerCache.states[name]``; the one without is ``LayerCache.state``)."""
    shape: Tuple[int, ...]
    dtype: str = "float32"
    name: str = ""


# ---- registries -----------------------------------------------------------

_KINDS: Dict[str, Dict[str, Callable]] = {
    "mixer": {}, "feed_forward": {}, "norm": {}, "position": {}, "qk_transform": {}, "block": {},
    "embedding": {}, "head": {}, "side_input": {}, "stream_entry": {},
}


def register_part(family: str, kind: str, factory: Callable) -> None:
    """``factory(spec: PartSpec, env: BuildEnv)`` returns the part.  ``family`` is one
    of mixer, feed_forward, norm, position, qk_transform, block, embedding, head, side_input, stream_entry."""
    if family not in _KINDS:
        raise KeyError(f"unknown part family {family!r}; families: {sorted(_KINDS)}")
    _KINDS[family][kind] = factory


def part_factory(family: str, kind: str) -> Callable:
    try:
        return _KINDS[family][kind]
    except KeyError:
        raise KeyError(f"no {family} of kind {kind!r} is registered; known: "
                       f"{sorted(_KINDS.get(family, {}))}") from None


@dataclass
class BuildEnv:
    """What every part is given at construction."""
    dtype: "object"      # torch.dtype of weights, activations and cache
    device: "object"     # torch.device
    hidden_size: int
    max_position: int
