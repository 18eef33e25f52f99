"""Data that describes a model: which parts, with which sizes, run in which order.

A model here is not a class per architecture but a `ModelSpec`: an embedding, a
tuple of `LayerSpec` (each naming its block arrangement, mixer, feed-forward,
norms and the prefix of its tensor names), a `schedule` that says in which order
layers run (a layer may be named twice, or read another layer's cache), a final
norm and a head.  An architecture is a function from its typed configuration to
such a spec (`liteinfer_b200/config/registry.py`); the parts themselves never
learn which model they are in.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable, Mapping


@dataclass(frozen=True)
class TensorSpec:
    """One checkpoint tensor a part reads.

    kind: "weight" is kept in the engine's dtype (bfloat16 or float32); "int" is
    an integer table kept as int32; "f32" stays 32-bit whatever the engine dtype.
    init: how the random-weights mode draws it: "normal" (N(0, 0.02)),
    "ones_normal" (1 + N(0, 0.01)), "zeros", or a function `(shape, generator) ->
    float32 tensor` for a part whose parameters need a distribution of their own
    (a decay kept in log space, a gate that must be positive).
    A size that only the checkpoint knows is None in `shape` (the part reads it off the tensor it is bound to); the
    random-weights mode draws it as `free` wide.
    """

    shape: tuple[int | None, ...]
    kind: str = "weight"
    init: str | Callable[[tuple[int, ...], Any], Any] = "normal"
    free: int = 0

    def accepts(self, shape: tuple[int, ...]) -> bool:
        return len(shape) == len(self.shape) and all(want in (None, got) for got, want in zip(shape, self.shape))

    def drawn_shape(self) -> tuple[int, ...]:
        return tuple(self.free if n is None else n for n in self.shape)


@dataclass(frozen=True)
class PartSpec:
    """A part by registry kind plus its constructor parameters."""

    kind: str
    params: Mapping[str, Any] = field(default_factory=dict)

    def __hash__(self) -> int:  # params is a dict; specs are compared by identity of content
        return hash((self.kind, tuple(sorted((k, repr(v)) for k, v in self.params.items()))))


@dataclass(frozen=True)
class LayerSpec:
    """One layer: an arrangement (`block`) of a mixer, a feed-forward and norms.

    `prefixes` maps the role of each part in the block ("mixer", "feed_forward",
    "mixer_norm", "feed_forward_norm", ...) to the prefix of its tensor names in
    the checkpoint, e.g. {"mixer": "model.layers.3.self_attn."}.
    """

    block: str
    parts: Mapping[str, PartSpec]
    prefixes: Mapping[str, str]
    # Per role, {the part's own name of a tensor: its name behind the prefix in this checkpoint}, for checkpoints
    # that spell a tensor differently ("q_proj.weight" stored as "q"); names not listed are kept.
    renames: Mapping[str, Mapping[str, str]] = field(default_factory=dict)


@dataclass(frozen=True)
class ScheduleEntry:
    """One stop of the forward pass: run `layer`.  `cache_of` is the index of an
    earlier stop of the schedule whose cache this stop reads instead of keeping
    one of its own (None: its own); such a stop stores nothing.  `reenter`: before this stop the model's
    `reentry` part runs on the residual stream (with the embedding's output as its second input)."""

    layer: int
    cache_of: int | None = None
    reenter: bool = False


@dataclass(frozen=True)
class ModelSpec:
    vocab_size: int
    hidden_size: int
    embedding: PartSpec
    embedding_prefix: str
    layers: tuple[LayerSpec, ...]
    schedule: tuple[ScheduleEntry, ...]
    final_norm: PartSpec
    final_norm_prefix: str
    head: PartSpec
    head_prefix: str
    # Tensor names that may be absent from a checkpoint because they alias another
    # tensor (a tied head): {absent name: name it reads instead}.
    tied: Mapping[str, str] = field(default_factory=dict)
    # "float32": the residual stream is kept in 32-bit whatever the engine's dtype (the embedding's output is
    # widened, the norms read and write it in 32-bit); None: it has the engine's dtype.
    stream_dtype: str | None = None
    # With a "float32" stream: the embedding writes the 32-bit stream itself, in one kernel (it is not read again).
    widened_embedding: bool = False
    # A number n: the residual of a token is n 32-bit streams side by side in one row [n * hidden_size], started by
    # the embedding's `forward_streams` (n equal copies) and read by norms that know streams (`stream_rmsnorm`);
    # None: one residual of hidden_size numbers.
    stream_copies: int | None = None
    # A part that mixes the embedding's output back into the stream before the stops marked `reenter`.
    reentry: PartSpec | None = None
    reentry_prefix: str = ""
    # Renames of the tensors of the parts that belong to no layer: {"embedding" | "final_norm" | "head" |
    # "reentry": {the part's own name: its name behind the prefix}}.
    renames: Mapping[str, Mapping[str, str]] = field(default_factory=dict)
    # Checkpoint names that may be present although no part reads them.
    ignored: tuple[str, ...] = ()

    def __post_init__(self) -> None:
        if not self.schedule:
            raise ValueError("a model's schedule names no layer")
        if self.stream_dtype not in (None, "float32"):
            raise ValueError(f"stream_dtype {self.stream_dtype!r} is not supported; known: None, 'float32'")
        if self.stream_copies is not None and (self.stream_copies < 1 or self.reentry is not None):
            raise ValueError("stream_copies must be >= 1, and a model with residual streams has no reentry part")
        if self.widened_embedding and (self.stream_dtype is None or self.reentry is not None):
            raise ValueError("widened_embedding is of a 32-bit stream whose embedding is not mixed in again")
        for stop, entry in enumerate(self.schedule):
            if entry.reenter and self.reentry is None:
                raise ValueError(f"stop {stop} re-enters the stream, but the model names no reentry part")
            if not 0 <= entry.layer < len(self.layers):
                raise ValueError(f"schedule names layer {entry.layer}, but there are {len(self.layers)}")
            if entry.cache_of is not None:
                if not 0 <= entry.cache_of < stop:
                    raise ValueError(f"stop {stop} reads the cache of stop {entry.cache_of}, which is not an earlier stop")
                if self.schedule[entry.cache_of].cache_of is not None:
                    raise ValueError(f"stop {stop} reads the cache of stop {entry.cache_of}, which keeps none of its own")
