"""Architecture-neutral description of a model: what the parts are built from.

An architecture's typed configuration (for instance ``Qwen3Config``) turns
itself into a ``ModelSpec``.  Everything below the configuration layer
(parts, cache manager, step function, trace replay, bench) reads only the
spec, so a new architecture adds a configuration class and, where it needs
them, new parts; nothing else changes.

Every size and constant of a part travels in its spec.  A part never asks
which model it belongs to.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping


@dataclass(frozen=True)
class NormSpec:
    """A normalisation over the last dimension."""

    kind: str          # key in parts.NORMS, e.g. "rmsnorm"
    size: int
    eps: float
    weight: str        # full tensor name of the scale
    bias: str | None = None    # full tensor name of the shift, for norms that have one
    groups: int = 1    # equal consecutive parts of the row with a statistic of their own, for norms that have it


@dataclass(frozen=True)
class PositionSpec:
    """A position encoding applied to queries and keys inside a mixer."""

    kind: str          # key in parts.POSITION_ENCODINGS, e.g. "rope_neox" or "none"
    head_dim: int
    max_positions: int
    params: Mapping[str, Any] = field(default_factory=dict)   # e.g. {"theta": 1e6}


@dataclass(frozen=True)
class MixerSpec:
    """The token mixer of a layer (attention here).

    ``params`` holds everything the mixer kind needs (head counts, head size,
    window, the names of its tensors).  ``position`` is the encoding it applies.
    """

    kind: str          # key in parts.MIXERS, e.g. "attention"
    params: Mapping[str, Any]
    position: PositionSpec | None = None


@dataclass(frozen=True)
class FeedForwardSpec:
    kind: str          # key in parts.FEED_FORWARDS, e.g. "swiglu"
    params: Mapping[str, Any]


@dataclass(frozen=True)
class SideSpec:
    """What joins the stream behind a layer's mixer and feed-forward, made from the stream itself."""

    kind: str          # key in parts.SIDES, e.g. "token_gate"
    params: Mapping[str, Any]


@dataclass(frozen=True)
class LayerSpec:
    """One layer: which block arrangement, and the parts placed in it.

    ``norms`` holds the layer's norms under the names the block arrangement gives them: the pre-norm
    residual block wants "mixer" and "feed_forward"; an arrangement with norms after its parts as
    well would name four."""

    block: str         # key in parts.BLOCKS, e.g. "prenorm_residual"
    mixer: MixerSpec
    feed_forward: FeedForwardSpec | None      # None: a layer without a feed-forward (where the block allows it)
    norms: Mapping[str, NormSpec]
    block_params: Mapping[str, Any] = field(default_factory=dict)   # the arrangement's own constants
    side: SideSpec | None = None      # for arrangements that take one (``Block.takes_side``)


@dataclass(frozen=True)
class InputSpec:
    """What turns a step's token ids into the first hidden states (a table lookup here)."""

    kind: str          # key in parts.INPUTS, e.g. "embedding"
    params: Mapping[str, Any]


@dataclass(frozen=True)
class OutputSpec:
    """What turns the last hidden states of the wanted tokens into float32 logits."""

    kind: str          # key in parts.OUTPUTS, e.g. "norm_head"
    params: Mapping[str, Any]


@dataclass(frozen=True)
class LayerCall:
    """One entry of the run order.

    ``layer`` indexes ``ModelSpec.layers`` (a layer may be named twice: its
    weights run again).  ``cache`` names the cache this call's mixer uses;
    calls with equal ``cache`` share it.  Only a call with ``writes_cache``
    stores new entries; a call without it reads what an earlier call of the
    same step stored (a layer that reads another layer's cache).  A mixer that
    keeps several stores (its ``cache_spec`` returns a tuple: pages beside a
    fixed state, or the stores of mixers that run side by side) gets the first
    under ``cache`` and the others under ``extra_caches``, in that order.
    """

    layer: int
    cache: int
    writes_cache: bool = True
    extra_caches: tuple[int, ...] = ()

    @property
    def caches(self) -> tuple[int, ...]:
        return (self.cache, *self.extra_caches)


@dataclass(frozen=True)
class ModelSpec:
    architecture: str
    vocab_size: int
    hidden_size: int
    max_seq_len: int
    input: InputSpec
    layers: tuple[LayerSpec, ...]
    run_order: tuple[LayerCall, ...]
    output: OutputSpec
    eos_token_ids: tuple[int, ...] = ()
    ignorable_weights: tuple[str, ...] = ()   # names a checkpoint may carry that are not read

    @property
    def num_caches(self) -> int:
        return 1 + max(cache for call in self.run_order for cache in call.caches)

    def validate(self) -> None:
        from .errors import ConfigError

        if not self.layers or not self.run_order:
            raise ConfigError("a model needs at least one layer and one run-order entry")
        writers: dict[int, int] = {}
        for index, call in enumerate(self.run_order):
            if not 0 <= call.layer < len(self.layers):
                raise ConfigError(f"run_order[{index}] names layer {call.layer}, which does not exist")
            for cache in call.caches:
                if cache < 0:
                    raise ConfigError(f"run_order[{index}] has a negative cache id")
                if call.writes_cache:
                    if cache in writers:
                        raise ConfigError(
                            f"cache {cache} is written by run_order[{writers[cache]}] and run_order[{index}]")
                    writers[cache] = index
                elif cache not in writers:
                    raise ConfigError(f"run_order[{index}] reads cache {cache} before any call has written it")
        if sorted(writers) != list(range(self.num_caches)):
            raise ConfigError("cache ids must be 0..n-1, each written by exactly one call")
