"""Architecture-neutral description of a model: what the part builders consume.

An architecture's configuration class turns its own ``config.json`` keys into a
:class:`ModelSpec`.  From here on nothing knows which architecture it is: a layer is a
block arrangement (a registered kind) of a mixer, a feed-forward and norms, each a
:class:`PartSpec` with its sizes and constants, chosen layer by layer.  The order in which
layers run is data as well: a list of :class:`RunSpec` that may name a layer twice (the
weights are shared, each run has a cache of its own) or let a run read the cache that an
earlier run owns.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from types import MappingProxyType
from typing import Any, Mapping, Optional, Union


@dataclass(frozen=True)
class PartSpec:
    """A registered part kind and the parameters its constructor takes."""

    kind: str
    params: Mapping[str, Any] = field(default_factory=dict)

    def __post_init__(self) -> None:
        object.__setattr__(self, "params", MappingProxyType(dict(self.params)))

    def __hash__(self) -> int:
        return hash((self.kind, repr(sorted(self.params.items(), key=lambda item: item[0]))))


@dataclass(frozen=True)
class LayerSpec:
    """One layer: a block arrangement of parts and the checkpoint prefix of its tensors."""

    prefix: str        # e.g. "model.layers.3."
    block: PartSpec    # arrangement kind; its parameters name the mixer, feed-forward, norms


@dataclass(frozen=True)
class RunSpec:
    """One entry of the run order: which layer runs, and whose cache its mixer is handed.

    ``cache_of`` is the index of an earlier entry of the order that owns a cache; ``None``
    means this run owns its own (sized by what its mixer says it needs).  ``add_embedding``: right
    before this run the step's embedding rows (scaled as they entered the stream) are added to the
    residual stream once more - what a model does that runs a span of layers several times and feeds
    its input in again at the start of every further pass.  ``reenter``: right before this run the stream is replaced by
    ``W [x; x0]``, x being the stream and x0 the embedding output of the step's tokens, both ``width`` wide, W the model's
    ``reentry_name`` tensor ``[width, 2 width]`` - how a pass of a looped span is entered.
    """

    layer: int
    cache_of: Optional[int] = None
    add_embedding: bool = False
    reenter: bool = False


@dataclass(frozen=True)
class ModelSpec:
    width: int                        # residual stream width
    vocab_size: int
    max_positions: int
    embedding_name: str               # checkpoint name of the [vocab, width] table
    lm_head_name: Optional[str]       # None: the head shares the embedding table
    final_norm: PartSpec
    final_norm_prefix: str
    layers: tuple[LayerSpec, ...]
    order: tuple[Union[RunSpec, int], ...]
    eos_token_ids: tuple[int, ...] = ()
    ignored_tensors: tuple[str, ...] = ()   # checkpoint names that may be present and are not used
    embedding_scale: float = 1.0            # the embedding rows are multiplied by it as they enter the residual stream
    logit_scale: float = 1.0                # the logits are multiplied by it,
    logit_softcap: Optional[float] = None   # then, with a cap c, squashed to c * tanh(logit / c)
    streams: int = 1                        # copies of the residual stream (hyper-connections); all start as the embedding row
    position_name: Optional[str] = None     # checkpoint name of a learnt table [position_rows, width]: row p is added to the embedding of the token at position p
    position_rows: int = 0
    reentry_name: Optional[str] = None      # checkpoint name of the [width, 2 width] matrix that runs with ``reenter`` go through
    embedding_norm: Optional[PartSpec] = None   # the embedding rows go through this norm, and what it gives is the stream they start
    embedding_norm_prefix: str = ""

    def __post_init__(self) -> None:
        runs = tuple(run if isinstance(run, RunSpec) else RunSpec(int(run)) for run in self.order)
        object.__setattr__(self, "order", runs)
        object.__setattr__(self, "layers", tuple(self.layers))
        if not runs:
            raise ValueError("a model must run at least one layer")
        if any(run.reenter for run in runs) and (self.reentry_name is None or self.streams != 1):
            raise ValueError("a run that re-enters needs the model's reentry matrix and a residual stream of one copy")
        if self.embedding_norm is not None and (self.streams != 1 or self.position_name is not None or any(run.add_embedding for run in runs)):
            raise ValueError("a norm on the embedding goes with a residual stream of one copy, without learnt positions and rows added again")
        if self.position_name is not None and not 0 < self.max_positions <= self.position_rows:
            raise ValueError(f"{self.max_positions} positions, but the table of learnt positions has {self.position_rows} rows")
        for position, run in enumerate(runs):
            if not 0 <= run.layer < len(self.layers):
                raise ValueError(f"run {position} names layer {run.layer}, but there are {len(self.layers)} layers")
            if run.cache_of is not None:
                if not 0 <= run.cache_of < position:
                    raise ValueError(f"run {position} reads the cache of run {run.cache_of}, which is not an earlier run")
                if runs[run.cache_of].cache_of is not None:
                    raise ValueError(f"run {position} reads the cache of run {run.cache_of}, which owns none")
