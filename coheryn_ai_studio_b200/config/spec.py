"""Architecture-neutral description of a decoder: which parts make up each layer,
with what parameters, and in what order layers run.

A model configuration (for example :class:`Qwen2Config`) is translated into a
:class:`ModelSpec` by the function registered for its architecture name.  Everything
below the registry (parts, cache manager, step function, scheduler) sees only the
:class:`ModelSpec`; no part knows which model it is in.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Mapping, Optional, Tuple


@dataclass(frozen=True)
class PartSpec:
    """One part of a layer: ``kind`` selects the class from the part registry of its
    role (mixer, feed_forward, norm, position); ``params`` are its constructor
    arguments (sizes and constants, never read from a global)."""

    kind: str
    params: Dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    """A layer = an arrangement (how the parts are wired, e.g. pre-norm residual) over the parts
    that fill its slots.  ``parts`` maps a slot name of the arrangement (for the pre-norm block:
    ``mixer``, ``feed_forward``, ``mixer_norm``, ``feed_forward_norm``) to the part that fills it;
    which slots exist, which may stay empty and what role each has is the arrangement's business,
    so a block without a feed-forward, with four norms or with two mixers is another arrangement
    and nothing else.  ``position`` is handed to the layer's mixers.  ``prefix`` is the
    tensor-name prefix of the layer's weights (``model.layers.3``)."""

    prefix: str
    arrangement: str
    parts: Mapping[str, PartSpec]
    position: Optional[PartSpec] = None
    # Slot name -> the component of the checkpoint's tensor names that the slot's part goes by, for an
    # arrangement whose checkpoints do not all use the same names (None: the arrangement's own).
    names: Optional[Mapping[str, str]] = None
    # Constants of the arrangement itself (its constructor's keyword arguments), e.g. the factor of the stream in a
    # block that normalises after the sum.
    arrangement_params: Mapping[str, Any] = field(default_factory=dict)


def prenorm_layer(prefix: str, mixer: PartSpec, feed_forward: PartSpec, mixer_norm: PartSpec,
                  feed_forward_norm: PartSpec, position: Optional[PartSpec] = None) -> LayerSpec:
    """The usual block: x += mixer(norm(x)); x += feed_forward(norm(x))."""
    return LayerSpec(prefix, "prenorm_residual",
                     {"mixer": mixer, "feed_forward": feed_forward, "mixer_norm": mixer_norm,
                      "feed_forward_norm": feed_forward_norm}, position)


@dataclass(frozen=True)
class StreamInject:
    """Something done to the residual stream right before a schedule entry runs.  Added to it: the embedding
    output of the step's tokens once more (``embedding``), and row ``vector[1]`` of the tensor
    named ``vector[0]`` (a [rows, width] tensor of ``ModelSpec.extra_tensors``).  Or, instead, ``mix``: the stream is
    REPLACED by M [x ; x0], x being the stream (with everything pending added), x0 the embedding output of the step's
    tokens and M the [width, 2 width] tensor of ``ModelSpec.extra_tensors`` that ``mix`` names."""

    embedding: bool = False
    vector: Optional[Tuple[str, int]] = None
    mix: Optional[str] = None


@dataclass(frozen=True)
class ScheduleEntry:
    """One execution of a layer.  The schedule is a list of these: a layer may be
    named twice (it then runs twice with the same weights, each run with a cache of
    its own), and ``cache_from`` lets an entry read the cache that an EARLIER entry
    of the schedule wrote instead of owning one.  ``inject`` is added to the stream
    before the entry runs (a model that repeats a span of its layers marks the start
    of each pass this way).  ``average``: with X_0 the embedding output and X_(j+1) the
    result of entry j, what entry i hands on is sum_j w[j] X_j over j = 0 .. i + 1, w being
    the tensor of ``ModelSpec.extra_tensors`` ([i + 2]) that ``average`` names."""

    layer: int
    cache_from: Optional[int] = None
    inject: Optional[StreamInject] = None
    average: Optional[str] = None


@dataclass(frozen=True)
class ModelSpec:
    architecture: str
    hidden_size: int
    vocab_size: int
    max_positions: int
    embedding_name: str
    layers: List[LayerSpec]
    schedule: List[ScheduleEntry]
    final_norm: PartSpec
    final_norm_name: str
    head_name: Optional[str]  # None: logits use the embedding table (tied)
    # Options that some architectures have and this one leaves at "none": the embedding rows are
    # multiplied by ``embedding_scale``; the logits are multiplied by ``logit_scale`` and a bias
    # ``head_bias_name`` (full tensor name, [vocab]) is added to them.
    embedding_scale: Optional[float] = None
    logit_scale: Optional[float] = None
    head_bias_name: Optional[str] = None
    # logits <- cap * tanh(logits / cap), after scale and bias.
    logit_softcap: Optional[float] = None
    # True: ``embedding_name``, ``head_name`` and ``final_norm_name`` are the tensors' full names
    # (no ".weight" is appended).
    bare_tensor_names: bool = False
    # Tensors of the model itself (not of a part): full name -> (shape, role, init) as for a TensorSpec.
    extra_tensors: Mapping[str, Tuple] = field(default_factory=dict)
    # The part that makes the stream from the step's token ids when a table row is not all of it (None: row
    # ``embedding_name`` of the table times ``embedding_scale``).  It names its tensors in full and owns the table.
    embedder: Optional[PartSpec] = None

    def validate(self) -> None:
        if not self.layers:
            raise ValueError("a model needs at least one layer")
        if not self.schedule:
            raise ValueError("the schedule names no layer")
        for i, e in enumerate(self.schedule):
            if not 0 <= e.layer < len(self.layers):
                raise ValueError(f"schedule entry {i} names layer {e.layer}, "
                                 f"but there are {len(self.layers)} layers")
            if e.cache_from is not None:
                if not 0 <= e.cache_from < i:
                    raise ValueError(
                        f"schedule entry {i} reads the cache of entry {e.cache_from}, "
                        "which is not an earlier entry")
                if self.schedule[e.cache_from].cache_from is not None:
                    raise ValueError(
                        f"schedule entry {i} reads the cache of entry {e.cache_from}, "
                        "which owns no cache itself")
            if e.average is not None and i and self.schedule[i - 1].average is None:
                raise ValueError(f"schedule entry {i} averages over depth and the entry before it does not: not built")
            if e.average is not None and tuple(self.extra_tensors.get(e.average, ((),))[0]) != (i + 2,):
                raise ValueError(f"schedule entry {i} averages over depth by {e.average!r}, which is not a [{i + 2}] tensor of "
                                 "the model")
            if e.inject is not None and e.inject.mix is not None:
                if e.inject.embedding or e.inject.vector is not None:
                    raise ValueError(f"schedule entry {i}: the stream is either replaced by a mix or added to, not both")
                shape = self.extra_tensors.get(e.inject.mix, (None,))[0]
                if shape is None or tuple(shape) != (self.hidden_size, 2 * self.hidden_size):
                    raise ValueError(f"schedule entry {i} mixes the stream by {e.inject.mix!r}, which is not a "
                                     f"[{self.hidden_size}, {2 * self.hidden_size}] tensor of the model")
                if self.embedder is not None:
                    raise ValueError(f"schedule entry {i}: a mix with the embedding output needs the plain embedding")
            if e.inject is not None and e.inject.vector is not None:
                name, row = e.inject.vector
                shape = self.extra_tensors.get(name, (None,))[0]
                if shape is None or len(shape) != 2 or shape[1] != self.hidden_size or not 0 <= row < shape[0]:
                    raise ValueError(f"schedule entry {i} adds row {row} of {name!r}, which is not a row of a "
                                     f"[rows, {self.hidden_size}] tensor of the model")
