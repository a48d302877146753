"""Data that describes a model: which parts make up each layer, and in which order layers run.

An architecture module turns its configuration into a :class:`ModelSpec`.  Everything in it
is data: part kinds are registry keys, sizes and constants are arguments, tensor names are
strings.  The model assembled from it (:mod:`.model`) knows no architecture.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Sequence


@dataclass(frozen=True)
class PartSpec:
    """A part chosen by ``kind`` (a key of the registry of its family) with its arguments."""

    kind: str
    args: Mapping[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    """One layer: a block arrangement around a mixer and a feed-forward with their norms.

    ``prefix`` is prepended to every tensor name the layer's parts declare.
    """

    prefix: str
    mixer: PartSpec
    feed_forward: Optional[PartSpec]           # None: the layer has no feed-forward
    mixer_norm: PartSpec
    feed_forward_norm: Optional[PartSpec]      # None: the block has one norm (``parallel``)
    block: PartSpec = PartSpec("pre_norm")
    # norms of a sublayer's OUTPUT, before it is added to the stream (blocks that norm on both sides of a sublayer)
    mixer_post_norm: Optional[PartSpec] = None
    feed_forward_post_norm: Optional[PartSpec] = None


@dataclass(frozen=True)
class LayerRun:
    """One entry of the execution order: run layer ``layer``.

    ``cache_of`` is ``None`` when the run keeps a cache of its own (if its mixer needs one);
    otherwise it is the index of an earlier entry of the order whose cache this run reads
    without writing to it.  ``enters`` is ``None`` or a pair ``(transition, number)``: before this run the stream goes
    through ``ModelSpec.transitions[transition]``, for the ``number``-th time of the step (the first is 0).
    """

    layer: int
    cache_of: Optional[int] = None
    enters: Optional[tuple] = None


@dataclass(frozen=True)
class ModelSpec:
    vocab_size: int
    hidden_size: int
    embedding_name: str
    layers: Sequence[LayerSpec]
    order: Sequence[LayerRun]
    final_norm: PartSpec
    output_name: Optional[str]      # None: the output matrix is the embedding table (tied)
    max_positions: int
    # True where the architecture has no position limit of its own and `max_positions` is only the engine's bound:
    # without an explicit `max_model_len` a runtime then takes the size of its page pool as the limit.
    nominal_max_positions: bool = False
    # Names that may be present in a checkpoint without being used (a stored copy of a tied matrix, the norm of a
    # feed-forward that a layer does not have).
    optional_names: Sequence[str] = ()
    # Those of `optional_names` that are stored copies of the tied output matrix: where present they must equal the
    # embedding table bit for bit.
    tied_copies: Sequence[str] = ()
    # The frame around the layers: embeddings are multiplied by `embedding_scale` as they enter the residual
    # stream; logits are multiplied by `logit_scale` and then, with `logit_softcap` c, become c * tanh(logit / c).
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    logit_softcap: Optional[float] = None
    # Parts of the embedding family whose rows are added to the (scaled) token embeddings, each with a table of its own
    # and, where it looks back along the sequence, a state that the request carries.
    extra_embeddings: Sequence[PartSpec] = ()
    # Parts of the transition family: what happens to the stream between two layers, where ``LayerRun.enters`` says so.
    transitions: Sequence[PartSpec] = ()
