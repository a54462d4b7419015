"""The model as data: which parts, with which numbers, in which order.

An architecture turns its configuration into a :class:`ModelSpec`.  The spec
names a kind for every part (looked up in the part registries) together with
the sizes and constants that part needs, layer by layer, so one model may mix
different mixers and feed-forwards.  The order in which layers run is a list
of :class:`RunEntry`: it may name a layer twice, and an entry may read the
cache that another entry writes.  Nothing here knows what a Llama is.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from types import MappingProxyType
from typing import Any, Mapping, Optional, Tuple


@dataclass(frozen=True)
class PartSpec:
    """A part's registered kind and its parameters (plain numbers and nested specs)."""

    kind: str
    params: Mapping[str, Any] = field(default_factory=dict)

    def __post_init__(self):
        object.__setattr__(self, "params", MappingProxyType(dict(self.params)))

    def __getitem__(self, key: str) -> Any:
        try:
            return self.params[key]
        except KeyError:
            raise KeyError(f"part '{self.kind}' was given no parameter '{key}'") from None

    def get(self, key: str, default: Any = None) -> Any:
        return self.params.get(key, default)


def part(kind: str, **params: Any) -> PartSpec:
    return PartSpec(kind, params)


@dataclass(frozen=True)
class LayerSpec:
    """One layer's own weights: ``name`` is the prefix of the layer's tensors (``layers.3``),
    ``block`` the arrangement.  The block's parameters carry everything inside it as nested
    specs (mixers, feed-forwards, norms, however many and wherever the block kind puts them),
    just as a mixer carries its position encoding; nothing outside the block kind knows what a
    layer is made of."""

    name: str
    block: PartSpec


@dataclass(frozen=True)
class RunEntry:
    """One run of a layer.  ``cache_of`` names the run (its index in the run
    order) whose cache this run reads instead of writing one of its own.

    What may be added to the stream right before the run (a model that runs a span of layers
    several times starts every pass this way): ``add_embedding`` adds the embedding output (the
    stream as it was before the first run), ``add_row = (tensor, i)`` adds row ``i`` of a model-level
    ``[rows, dim]`` tensor (``ModelSpec.row_tensors``) to every token.  Both sums are 32-bit.
    ``join_embedding = tensor`` replaces the stream by a product first: with ``W`` the model-level ``[dim, 2 dim]``
    matrix of that name (``ModelSpec.join_tensors``), ``h <- W [h; embedding output]``; a row is added after it."""

    layer: int
    cache_of: Optional[int] = None
    add_embedding: bool = False
    add_row: Optional[Tuple[str, int]] = None
    join_embedding: Optional[str] = None


@dataclass(frozen=True)
class PairTable:
    """A table of rows by pairs of neighbouring tokens, added to the embedding: with ``p`` the request's token before
    ``t``, row ``(p * mul_prev + t * mul_cur) mod buckets`` of the model-level ``[buckets + 1, dim]`` tensor; a request's
    first token, which has none before it, takes the last row.  The last token of every request is model-level state."""

    tensor: str
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class ModelSpec:
    dim: int
    vocab_size: int
    max_positions: int
    embedding_tensor: str            # name of the [vocab, dim] table
    layers: Tuple[LayerSpec, ...]
    run_order: Tuple[RunEntry, ...]
    final_norm: PartSpec
    final_norm_prefix: str           # prefix of the final norm's tensors
    head_tensor: str                 # name of the [vocab, dim] output matrix
    tie_head: bool = False           # the head is the embedding table; head_tensor is absent
    embedding_scale: float = 1.0     # the rows of the table enter the stream multiplied by this
    position_tensor: Optional[str] = None   # name of a learned [max_positions, dim] table added to the embedding
    keeps_history: bool = False      # the result of every layer run stays readable by later runs (Residual.history)
    embedding_norm: Optional[PartSpec] = None        # a norm applied to the table's row: its result is the stream
    embedding_norm_prefix: str = "embedding_norm"    # prefix of that norm's tensors
    logit_scale: float = 1.0         # the head's products leave multiplied by this
    row_tensors: Tuple[Tuple[str, int], ...] = ()    # model-level (name, rows) tensors [rows, dim] whose rows runs add to the stream (RunEntry.add_row)
    pair_table: Optional[PairTable] = None           # rows by pairs of neighbouring tokens, added to the embedding
    join_tensors: Tuple[str, ...] = ()               # model-level [dim, 2 dim] matrices that join the stream and the embedding output (RunEntry.join_embedding)

    def __post_init__(self):
        n = len(self.layers)
        rows = dict(self.row_tensors)
        for i, run in enumerate(self.run_order):
            if run.add_row is not None and not (run.add_row[0] in rows and 0 <= run.add_row[1] < rows[run.add_row[0]]):
                raise ValueError(f"run {i} adds row {run.add_row[1]} of '{run.add_row[0]}', which the model does not have")
            if run.join_embedding is not None and (run.join_embedding not in self.join_tensors or run.add_embedding):
                raise ValueError(f"run {i} joins the embedding output through '{run.join_embedding}', which the model does not have, "
                                 "or adds it as well")
            if not 0 <= run.layer < n:
                raise ValueError(f"run {i} names layer {run.layer}, but there are {n} layers")
            if run.cache_of is not None:
                if not 0 <= run.cache_of < i:
                    raise ValueError(
                        f"run {i} reads the cache of run {run.cache_of}, which must come before it")
                if self.run_order[run.cache_of].cache_of is not None:
                    raise ValueError(
                        f"run {i} reads the cache of run {run.cache_of}, which owns none itself")
