"""Architecture-neutral description of a model: which parts, with which constants,
in which order.

A typed architecture configuration (for instance ``Qwen2Config``) is turned into a
``ModelSpec``; everything below the configuration layer (weights, parts, cache,
engine) reads only the ``ModelSpec``.  The reference passes the same constants as
constructor arguments layer by layer
(v10_triton_paged_gqa/layer/transformer_block.py:10-35); here they are data so that
layers may differ from one another and the run order is a list.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Optional


@dataclass(frozen=True)
class PartSpec:
    """One part of a layer: its registered kind and its own constants."""

    kind: str
    params: dict = field(default_factory=dict)

    def get(self, key: str, default: Any = None) -> Any:
        return self.params.get(key, default)


@dataclass(frozen=True)
class NormSlot:
    """One norm of a layer: the role the block arrangement knows it by (for instance
    "mixer_norm"), its part, and the tensor-name prefix of its weights below the layer's."""

    role: str
    part: PartSpec
    prefix: str


@dataclass(frozen=True)
class LayerSpec:
    """One layer's parts and where their tensors are found.

    ``prefix`` is the tensor-name prefix of the layer; each part's tensors lie below
    ``prefix + <part prefix>``.  The part prefixes are the checkpoint's own names, set by the
    architecture's configuration; nothing below the configuration layer spells one out.
    ``norms`` holds as many norms as the block arrangement ``block`` asks for, by role.
    ``feed_forward`` may be None (a layer of a mixer alone).  ``block_params`` are the
    arrangement's own constants (a residual multiplier, for instance).  ``token_input`` is an
    optional part that adds something computed from the token ids themselves after the layer's
    sub-layers (a per-layer token embedding).
    """

    prefix: str
    block: str  # arrangement of the parts, e.g. "pre_norm"
    mixer: PartSpec
    feed_forward: Optional[PartSpec]
    norms: tuple = ()  # of NormSlot
    mixer_prefix: str = "mixer."
    feed_forward_prefix: str = "feed_forward."
    block_params: dict = field(default_factory=dict)
    token_input: Optional[PartSpec] = None
    token_input_prefix: str = "token_input."

    def norm(self, role: str) -> NormSlot:
        for slot in self.norms:
            if slot.role == role:
                return slot
        raise KeyError(f"layer {self.prefix!r} has no norm for the role {role!r}; "
                       f"it has: {', '.join(s.role for s in self.norms) or 'none'}")


@dataclass(frozen=True)
class ScheduleEntry:
    """One execution of a layer.

    ``layer`` indexes ``ModelSpec.layers`` and may appear more than once in the
    schedule.  Each entry owns the cache of its execution unless ``cache_from``
    names an earlier entry, whose cache it then reads without writing.  ``add_embedding``: before this
    execution the embedding output (the stream as it entered the first layer) is added to the stream
    (a model that runs a stretch of its layers several times feeds its input in again before each
    further pass).  ``add_row`` = r: row r of the table ``ModelSpec.stream_rows_name`` is added to every token's stream
    before this execution (a vector that tells the passes of a looped stretch apart).
    """

    layer: int
    cache_from: Optional[int] = None
    add_embedding: bool = False
    add_row: Optional[int] = None


@dataclass(frozen=True)
class TokenPairs:
    """A second embedding table whose row is chosen by a token AND the one before it in its sequence: row
    (previous * ``mul_prev`` + token * ``mul_cur``) mod ``buckets`` of ``table_name`` [buckets + 1, hidden]; the last row
    is that of a sequence's first token.  The row is added to the token's embedding (before an embedding norm); every
    request's last token is therefore state."""

    table_name: str
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class ModelSpec:
    architecture: str
    vocab_size: int
    hidden_size: int
    max_position_embeddings: int
    embedding_name: str
    layers: tuple
    schedule: tuple
    final_norm: PartSpec
    final_norm_prefix: str
    lm_head_name: str
    tie_word_embeddings: bool
    embedding_scale: float = 1.0  # the stream starts as embedding[token] * embedding_scale
    logit_scale: float = 1.0  # logits = (head . normed stream) * logit_scale
    # None: one residual stream [T, hidden].  n >= 1: the blocks work on n streams a token, [T, n, hidden], which all
    # start as the embedding output and are summed before the final norm (every block must be of such a kind).
    streams: Optional[int] = None
    # a norm of the embedding rows (after the scale) before the first layer; its tensors lie below the prefix
    embedding_norm: Optional[PartSpec] = None
    embedding_norm_prefix: str = "embedding_norm."
    # a tensor [stream_rows, hidden] whose rows schedule entries add to the stream (``ScheduleEntry.add_row``)
    stream_rows_name: Optional[str] = None
    stream_rows: int = 0
    token_pairs: Optional[TokenPairs] = None  # a row for every pair of neighbouring tokens, added to the embedding

    def validate(self) -> None:
        if not self.layers:
            raise ValueError("a model needs at least one layer")
        if not self.schedule:
            raise ValueError("the layer schedule is empty")
        if self.streams is not None and any(entry.add_embedding for entry in self.schedule):
            raise ValueError("adding the embedding output again is not built for several residual streams")
        if self.streams is not None and any(entry.add_row is not None for entry in self.schedule):
            raise ValueError("adding a row to the stream is not built for several residual streams")
        for i, entry in enumerate(self.schedule):
            if entry.add_row is not None and (self.stream_rows_name is None or not 0 <= entry.add_row < self.stream_rows):
                raise ValueError(f"schedule entry {i} adds row {entry.add_row} of a table of {self.stream_rows} rows")
            if not 0 <= entry.layer < len(self.layers):
                raise ValueError(
                    f"schedule entry {i} names layer {entry.layer}, "
                    f"but there are {len(self.layers)} layers"
                )
            if entry.cache_from is not None:
                if not 0 <= entry.cache_from < i:
                    raise ValueError(
                        f"schedule entry {i} reads the cache of entry {entry.cache_from}, "
                        "which must be an earlier entry"
                    )
                if self.schedule[entry.cache_from].cache_from is not None:
                    raise ValueError(
                        f"schedule entry {i} reads the cache of entry {entry.cache_from}, "
                        "which owns no cache itself"
                    )
