"""The description of a model as data: which parts make each layer, in which order the layers
run and which cache each run of a layer reads and writes.

An architecture's ``build_plan(config)`` returns a :class:`ModelPlan`; nothing below this file
knows which architecture it serves.  The reference wires one fixed stack instead
(``ginfer/model/model.cc:34-46``: embedding, ``nlayer`` identical ``EncoderLayer``s, final
RMSNorm, LM head); the plan generalises that stack so that layers may differ and the run order
is a list.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping


@dataclass(frozen=True)
class PartSpec:
    """A part by registered kind, with its sizes and constants as parameters."""
    kind: str
    params: Mapping[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    """One layer: an arrangement (``block``) of a mixer, a feed-forward and their norms.
    ``prefix`` is the tensor-name prefix of the layer (``model.layers.3``).  A layer without a
    feed-forward has ``None`` for it and its norm (blocks that allow it say so)."""
    prefix: str
    mixer: PartSpec
    feed_forward: PartSpec | None
    mixer_norm: PartSpec
    feed_forward_norm: PartSpec | None
    block: PartSpec = PartSpec("prenorm")


@dataclass(frozen=True)
class RunEntry:
    """One run of a layer.  ``layer`` indexes :attr:`ModelPlan.layers` (a layer may be named
    twice).  ``cache`` names the cache this run uses: by default a cache of its own; a run with
    ``write_cache=False`` only reads the cache another run has written earlier in the step.  A mixer
    made of several names a cache for each, in their order (a tuple).
    ``enter = (i, n)``: before this run the stream passes through
    :attr:`ModelPlan.stream_inputs` ``[i]`` as its entry number ``n`` (the start of a pass of a
    loop, say).  ``block_state`` names the per-request state of the layer's block itself, beside
    its mixer's cache (for blocks that keep one)."""
    layer: int
    cache: int | tuple[int, ...]
    write_cache: bool = True
    enter: tuple[int, int] | None = None
    block_state: int | None = None

    def caches(self) -> tuple[int, ...]:
        return self.cache if isinstance(self.cache, tuple) else (self.cache,)


@dataclass(frozen=True)
class ModelPlan:
    hidden_size: int
    vocab_size: int
    max_positions: int
    embedding: PartSpec
    layers: tuple[LayerSpec, ...]
    run: tuple[RunEntry, ...]
    final_norm: PartSpec
    head: PartSpec
    eos_token_ids: tuple[int, ...] = ()
    stream_inputs: tuple[PartSpec, ...] = ()   # parts that runs enter through (RunEntry.enter)
    embedding_state: int | None = None   # the per-request state of the embedding, if it keeps one
    ignored_tensors: tuple[str, ...] = ()     # regular expressions of tensor names to pass over

    def validate(self) -> None:
        writers: dict[int, int] = {}
        for pos, e in enumerate(self.run):
            if not (0 <= e.layer < len(self.layers)):
                raise ValueError(f"run[{pos}] names layer {e.layer}, but there are "
                                 f"{len(self.layers)} layers")
            if e.enter is not None and not (0 <= e.enter[0] < len(self.stream_inputs)):
                raise ValueError(f"run[{pos}] enters through stream input {e.enter[0]}, but "
                                 f"there are {len(self.stream_inputs)}")
            for c in e.caches() if e.write_cache else ():
                if c in writers:
                    raise ValueError(f"run[{pos}] and run[{writers[c]}] both write cache {c}")
                writers[c] = pos
            if e.block_state is not None:
                if e.block_state in writers:
                    raise ValueError(f"run[{pos}] keeps its block's state as {e.block_state}, "
                                     f"which run[{writers[e.block_state]}] writes")
                writers[e.block_state] = pos
        for pos, e in enumerate(self.run):
            for c in () if e.write_cache else e.caches():
                if c not in writers or writers[c] > pos:
                    raise ValueError(f"run[{pos}] reads cache {c} before any run writes it")
        if self.embedding_state is not None and self.embedding_state in writers:
            raise ValueError(f"the embedding keeps its state as {self.embedding_state}, which "
                             f"run[{writers[self.embedding_state]}] writes")


def sequential_run(num_layers: int) -> tuple[RunEntry, ...]:
    """Every layer once, in order, each with a cache of its own."""
    return tuple(RunEntry(layer=i, cache=i) for i in range(num_layers))
