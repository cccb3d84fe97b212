"""Plain data that describes a model: which parts each layer is made of, and the order layers run in.

A model is data before it is code.  An architecture's builder turns its typed
configuration into a :class:`ModelSpec`; :class:`marin_b200.models.model.Model` turns the
spec into parts by looking every ``kind`` up in the part registries.  Nothing in
a part knows which model it is in: it sees only its own parameters.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple


@dataclass(frozen=True)
class TensorSpec:
    """One tensor a part expects in the checkpoint.

    ``role`` decides storage and random initialisation: ``matrix`` (bf16 or f32,
    N(0, 0.02)), ``norm`` (kept f32 on the device, 1 + N(0, 0.05)), ``bias`` (kept f32 on
    the device, N(0, 0.02): offsets, mixing coefficients, small tables added to scores),
    ``table`` (an embedding table, treated like a matrix), ``int_table`` (int32).  ``mean`` moves the centre of the random
    initialisation (a mixing coefficient that should start near 1 or near 1/n rather than near 0).  ``limit`` (integer
    tables): entries are drawn below it, those of a row all different (a table that names a token's experts).
    """

    name: str
    shape: Tuple[int, ...]
    role: str = "matrix"
    mean: Optional[float] = None
    limit: Optional[int] = None


@dataclass
class PartSpec:
    """A part chosen by name from a registry, with the parameters it is built from."""

    kind: str
    params: Dict[str, Any] = field(default_factory=dict)


@dataclass
class LayerSpec:
    """One layer: how its parts are arranged (``block``) and which parts they are."""

    block: str
    norm: PartSpec
    mixer: PartSpec
    #: None: the layer has no feed-forward sublayer (and no second norm)
    feedforward: Optional[PartSpec]
    prefix: str
    #: names inside ``prefix`` of the sub-modules, so that parts find their tensors
    names: Dict[str, str] = field(default_factory=dict)
    #: what the block arrangement itself is built from, besides its parts (a hyper-connection block: the number of streams)
    block_params: Dict[str, Any] = field(default_factory=dict)


@dataclass
class ScheduleEntry:
    """One run of a layer.  ``cache_of`` names an earlier entry whose cache this run reads
    instead of keeping one of its own (it then writes nothing).  ``enters``: this run starts pass ``enters`` of a loop: the pass's row of
    ``ModelSpec.pass_vectors`` is added to the stream right before it, and before that, in every pass but the first, the embedding's output."""

    layer: int
    cache_of: Optional[int] = None
    enters: Optional[int] = None


@dataclass
class ModelSpec:
    hidden_size: int
    vocab_size: int
    embedding: PartSpec
    final_norm: PartSpec
    head: PartSpec
    layers: List[LayerSpec]
    schedule: List[ScheduleEntry]
    #: tensors that may be present in a checkpoint and are ignored (e.g. an unused head when tied)
    ignorable: Tuple[str, ...] = ()
    #: how many copies of the residual stream the blocks keep (hyper-connections): the model then hands its blocks a float32
    #: ``[streams, T, hidden]`` tensor (also for a single copy) and the head reads their sum; 0: one plain ``[T, hidden]`` stream
    streams: int = 0
    #: a tensor ``[passes, hidden]`` whose rows are added to the stream where passes start (``ScheduleEntry.enters``)
    pass_vectors: Optional[TensorSpec] = None
