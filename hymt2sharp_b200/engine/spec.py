"""The description of a model that the engine builds from: which parts make up
each layer, in which order the layers run, and where the embedding, the final
norm and the output head come from.  An architecture's builder turns its
configuration into this; nothing below it knows the architecture."""
from __future__ import annotations

from dataclasses import dataclass, field

from ..parts.base import PartSpec


@dataclass
class Bigram:
    """A second table whose rows belong to pairs of tokens: the embedding of `token` behind `previous` adds row
    (previous * mul_prev + token * mul_cur) mod buckets.  Where nothing stands in front (position 0) it adds the row behind the
    buckets.  Which token came last is kept with the sequence, in its state row."""
    table: str                        # checkpoint name of the [buckets + 1, hidden] table
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass
class Run:
    """One entry of the order in which layers run.  A layer may be named by several
    entries (it then runs several times with the same weights, each run with a cache
    plane of its own), and an entry may read the cache plane that an earlier entry
    wrote (`cache_from` = that entry's index in the order) instead of writing one.
    With `joins` the residual x becomes W [x; x0] before the layer runs, x0 being the
    embedding's output and W the matrix that the spec's `join` names; with `adds` it
    becomes x + x0."""
    layer: int
    cache_from: int | None = None
    joins: bool = False
    adds: bool = False


@dataclass
class ModelSpec:
    vocab: int
    hidden: int
    embedding: str                    # checkpoint name of the [vocab, hidden] table
    layers: list[PartSpec]            # block specs (category "block")
    final_norm: PartSpec
    head: str | None                  # checkpoint name of the [vocab, hidden] head; None = the embedding table
    order: list[Run] = field(default_factory=list)
    max_positions: int | None = None  # the longest sequence the model takes (None: whatever the cache holds)
    embed_scale: float | None = None  # the embedding rows are multiplied by this (None: as they are)
    logit_scale: float | None = None  # the logits are multiplied by this (None: as they are)
    logit_softcap: float | None = None  # the logits become cap * tanh(logits / cap) (None: as they are)
    # regular expressions of tensor names that checkpoints of this architecture may hold and the model does not read
    ignorable_tensors: list[str] = field(default_factory=list)
    head_copy: str | None = None      # with a tied head: the name under which a checkpoint may store the head once more
    # None: the residual is one matrix [T, hidden].  n >= 1: it is kept as n streams [n, T, hidden] (parts.block.StreamsBlock),
    # all equal to the embedding's output at the start and added up in front of the final norm
    residual_streams: int | None = None
    bigram: Bigram | None = None      # (None: the embedding's rows alone)
    join: str | None = None           # checkpoint name of the [hidden, 2 hidden] matrix of the runs that say `joins`
    positions: str | None = None      # checkpoint name of a [max_positions, hidden] table: row p is added at position p (not scaled)

    def __post_init__(self):
        if not self.order:
            self.order = [Run(i) for i in range(len(self.layers))]
        if any(run.joins for run in self.order) and (self.join is None or self.residual_streams is not None):
            raise ValueError("a run that joins the residual with the embedding's output needs the matrix's name and one residual stream")
        if any(run.adds for run in self.order) and (self.residual_streams is not None or self.order[0].adds):
            raise ValueError("the embedding's output is added to a residual in one stream, behind the first run")
        if any(run.adds and run.joins for run in self.order):
            raise ValueError("a run either joins the residual with the embedding's output or adds it")
        if self.positions is not None and (self.max_positions is None or self.bigram is not None or self.residual_streams is not None):
            raise ValueError("a table of positions comes with its length, without a table of pairs and with one residual stream")
        for i, run in enumerate(self.order):
            if not (0 <= run.layer < len(self.layers)):
                raise ValueError(f"order[{i}] names layer {run.layer}, the model has {len(self.layers)}")
            if run.cache_from is not None:
                if not (0 <= run.cache_from < i):
                    raise ValueError(f"order[{i}] reads the cache of entry {run.cache_from}, which does not run before it")
                if self.order[run.cache_from].cache_from is not None:
                    raise ValueError(f"order[{i}] reads the cache of entry {run.cache_from}, which has none of its own")
