"""Plain data that describes a model: which parts, with which constants, in which order.

A ``ModelSpec`` is what an architecture's ``describe(config)`` returns. Nothing in it
is executable: parts are named by kind and looked up in the part registries when the
model is built, so a model may use a different mixer or feed-forward in every layer.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable, Mapping


@dataclass(frozen=True)
class PartSpec:
    """One part: its registered kind, its sizes and constants, and the prefix (relative
    to the layer's prefix) under which its tensors are stored. ``names`` maps the part's
    own tensor names to other stored names where an architecture calls them differently."""

    kind: str
    params: Mapping[str, Any] = field(default_factory=dict)
    prefix: str = ""
    names: Mapping[str, str] = field(default_factory=dict)

    def __getitem__(self, key: str) -> Any:
        return self.params[key]

    def get(self, key: str, default: Any = None) -> Any:
        return self.params.get(key, default)

    def stored_name(self, local: str) -> str:
        return self.prefix + self.names.get(local, local)


class FreeSize(int):
    """A size that the stored tensor decides (an inner size that config.json does not give).
    ``name`` ties sizes together: within a layer's part every dimension with that name has the
    same size. The number itself is what the random-weights mode uses."""

    def __new__(cls, name: str, default: int):
        size = super().__new__(cls, default)
        size.name = name
        return size

    def within(self, prefix: str) -> "FreeSize":
        return FreeSize(prefix + self.name, int(self))


@dataclass(frozen=True)
class TensorSpec:
    """Shape of a stored tensor and how the random-weights mode fills it:
    ``normal`` ~ N(0, std), ``norm`` ~ 1 + N(0, 0.1), ``bias`` ~ N(0, std), ``norm0`` ~
    N(0, 0.1) (a norm weight stored around zero), ``wide`` ~ N(0, 0.5), ``mix`` (a square matrix
    near the identity) ~ 1 + N(0, 0.1) on the diagonal and N(0, 0.1) beside it."""

    shape: tuple[int, ...]
    init: str = "normal"

    def within(self, prefix: str) -> "TensorSpec":
        """The same with its free sizes' names made unique to the part stored under ``prefix``."""
        if not any(isinstance(size, FreeSize) for size in self.shape):
            return self
        return TensorSpec(tuple(size.within(prefix) if isinstance(size, FreeSize) else size
                                for size in self.shape), self.init)

    def fits(self, shape, sizes: dict[str, int]) -> bool:
        """Whether a stored tensor of ``shape`` is what is wanted. ``sizes`` keeps the free sizes
        met so far, by name."""
        if len(shape) != len(self.shape):
            return False
        for got, want in zip(shape, self.shape):
            if isinstance(want, FreeSize):
                want = sizes.setdefault(want.name, int(got)) if got > 0 else -1
            if got != want:
                return False
        return True


@dataclass(frozen=True)
class LayerSpec:
    """One layer: a block arrangement and the parts it arranges, by role. A layer without a
    feed-forward has ``feed_forward`` and ``feed_forward_norm`` None."""

    prefix: str
    block: PartSpec
    mixer: PartSpec
    mixer_norm: PartSpec
    feed_forward: PartSpec | None
    feed_forward_norm: PartSpec | None


@dataclass(frozen=True)
class Injection:
    """Something added to every token's residual stream right before a call of the order:
    row ``row`` of the stored tensor ``vector`` ([rows, hidden], listed in
    ``ModelSpec.vectors``), and, with ``embedding``, the token's embedding once more.
    With ``mix`` (the stored name of a [hidden, 2 hidden] matrix, also listed in
    ``ModelSpec.vectors``) the stream is first replaced by that matrix applied to the stream and
    the token's embedding side by side (stream first); the vector's row is added to the result."""

    vector: str | None = None
    row: int = 0
    embedding: bool = False
    mix: str | None = None


@dataclass(frozen=True)
class LayerCall:
    """One entry of the execution order. ``layer`` indexes ``ModelSpec.layers`` and may
    appear more than once. ``cache`` names the cache entry that the call's mixer uses;
    by default every call has an entry of its own (its index in the order). A call with
    ``writes_cache=False`` reads an entry that an earlier call of the step has written.
    ``inject`` is added to the stream before the call (a loop's pass that starts here)."""

    layer: int
    cache: int | None = None
    writes_cache: bool = True
    inject: Injection | None = None


@dataclass(frozen=True)
class ModelSpec:
    architecture: str
    vocab_size: int
    hidden_size: int
    embedding: str                          # stored name of the [vocab, hidden] table
    layers: tuple[LayerSpec, ...]
    order: tuple[LayerCall, ...]
    final_norm: PartSpec
    head: str | None                        # stored name of the output matrix; None = tied
    max_positions: int
    eos_token_ids: tuple[int, ...] = ()
    bos_token_id: int | None = None
    init_std: float = 0.02
    # (stored name, shape) -> (name, squeeze axis or None), or None to drop the tensor
    rename: Callable[[str, tuple[int, ...]], tuple[str, int | None] | None] | None = None
    # stored tensors that belong to no part (what ``Injection.vector`` names): name -> TensorSpec
    vectors: Mapping[str, Any] = field(default_factory=dict)
    # logits become cap * tanh(logits / cap); None: the output product's values as they are
    logit_softcap: float | None = None
    # a factor on the output product's values (applied before a cap)
    logit_scale: float = 1.0
    # an embedding part (registry EMBEDDINGS) that makes the stream's first value; None: row
    # ``token`` of the table ``embedding``. Its table is stored under ``embedding`` all the same.
    embedding_part: PartSpec | None = None
