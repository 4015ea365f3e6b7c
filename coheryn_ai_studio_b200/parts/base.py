"""Interfaces of the parts a layer is assembled from, and the registries that map a
:class:`PartSpec` kind to a class.

A part is built from its parameters alone (``cls(**spec.params)`` plus the runtime's
dtype and device); it names the tensors it wants (:meth:`Part.tensor_specs`), receives
them (:meth:`Part.bind`) and runs on the device.  Roles:

* mixer         – ``forward(x, step, cache) -> y``; moves information between the tokens
                  of a request; says what cache it needs (:meth:`Mixer.cache_requirement`).
* feed_forward  – ``forward(x, step) -> y``; token-wise.
* norm          – ``forward(residual, delta, out_rows=None) -> normed``; adds ``delta`` to
                  the float32 residual stream in place and normalises.
* position      – owns what a mixer needs to encode positions (here: a rotation table).
* arrangement   – wires mixer, feed-forward and norms into a block.

New kinds are added with the ``register_*`` functions; nothing else has to change.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from ..config.spec import PartSpec
from ..weights.spec import TensorSpec


@dataclass(frozen=True)
class Runtime:
    """Where and in which precision the parts run."""

    dtype: torch.dtype            # torch.float32 or torch.bfloat16: activations, matrices, cache
    device: torch.device


# ------------------------------------------------------------------ cache requirements
@dataclass(frozen=True)
class PagedKV:
    """Keys and values of every position (``window`` None) or of the last ``window``
    positions, kept in pages."""

    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    v_head_dim: Optional[int] = None      # values of another head size than keys (None: the same; 0: no value rows at
                                          # all, the mixer finds its values inside the key rows)
    stride: int = 1                       # one row for every ``stride`` positions (a summary of a block of positions): a
                                          # page then has ceil(page_size / stride) rows, under a block table of its own;
                                          # the block whose LAST position is p lives in p's page, at row
                                          # block - floor(page * page_size / stride)

    keep_first: int = 0                   # with a window: the first positions of a sequence, which stay visible (and cached)
                                          # although the window has passed them

    def rows_per_page(self, page_size: int) -> int:
        return -(-page_size // self.stride)

    @property
    def value_dim(self) -> int:
        """Channels of a value row as the pool keeps it."""
        return self.head_dim if self.v_head_dim is None else self.v_head_dim


@dataclass(frozen=True)
class FixedState:
    """State of fixed size per request, zeroed when the request is admitted."""

    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass
class LayerCache:
    """What a mixer gets for one execution of its layer.

    Paged: ``k``/``v`` are ``[pages, kv heads, page_size, head_dim]`` views of the
    group's pool for this schedule entry; ``group`` indexes ``step.block_tables`` and
    ``step.slots``; ``writes`` is False when the entry reads another entry's cache.
    Fixed state: ``state`` is ``[slots, *shape]``; ``step.state_slots`` gives each
    request's slot."""

    kind: str                      # "paged" | "state" | "several"
    group: int = -1
    page_size: int = 0
    k: Optional[torch.Tensor] = None
    v: Optional[torch.Tensor] = None
    writes: bool = True
    state: Optional[torch.Tensor] = None
    # "several": a mixer that asked for a tuple of requirements gets one cache per element, in order.
    parts: Optional[List["LayerCache"]] = None


@dataclass
class StepContext:
    """One batch of (request, its next tokens) as the device sees it.  Requests are
    numbered 0..B-1 in the order of the batch; their tokens are laid out one request
    after the other."""

    num_tokens: int
    num_requests: int
    token_ids: torch.Tensor           # [T] int32
    positions: torch.Tensor           # [T] int32, absolute position of each token
    token_req: torch.Tensor           # [T] int32, batch index of each token's request
    cu_q: torch.Tensor                # [B+1] int32, token offsets of the requests
    kv_lens: torch.Tensor             # [B] int32, tokens of each request after this step
    block_tables: List[torch.Tensor]  # per cache group: [B, max_blocks] int32
    slots: List[torch.Tensor]         # per cache group: [T] int32 page*page_size+offset
    state_slots: torch.Tensor         # [B] int32
    q_lens: List[int] = field(default_factory=list)       # host copies
    kv_lens_host: List[int] = field(default_factory=list)
    max_q_len: int = 0
    max_kv_len: int = 0
    # When few of the step's rows are wanted: the wanted rows as a step of their own (one row
    # per "request": one query at its position over the same pages) and their indices among the
    # step's tokens.  The LAST entry of the schedule then computes only these rows after it has
    # updated its cache for all of them (crates/coheryn-engine/src/inference.rs:481-485: a row
    # that needs no logits stops after the append in the last layer).  tail.num_tokens may be 0.
    tail: Optional["StepContext"] = None
    tail_rows: Optional[torch.Tensor] = None   # [R] int32
    # True (every ordinary step): what the cache holds at positions BEFORE a request's first token
    # of this step was written by earlier steps, so a kernel may read it ahead of the step's own
    # kernels.  False for the context of the wanted rows (``tail``): its one-token "requests" look
    # back on keys and values that this same step has just written.
    prior_positions_settled: bool = True
    # Scratch of parts/native_block.py: what the blocks of this step share once the first of them
    # has described the step to the library.
    native: Optional[object] = None
    # What a layer of this step leaves for later layers of the same step (for instance the values that later layers mix
    # into theirs), by a name the parts agree on; emptied when the model starts a step.
    shared: Dict[str, torch.Tensor] = field(default_factory=dict)


@dataclass
class NormedSum:
    """A producer's output that is a sum of normalised summands, not yet formed:
    y = coef * sum_p parts[p] / rms(parts[p]) * weights[p], rms over the last axis with ``eps`` inside the root.
    ``parts`` float32 [P, T, H], ``weights`` [P, H]."""

    parts: torch.Tensor
    weights: torch.Tensor
    coef: float
    eps: float

    def resolve(self) -> torch.Tensor:
        """The sum itself, by library operations (traces and tests; the product path hands the object on)."""
        p = self.parts.float()
        y = p * torch.rsqrt((p * p).mean(-1, keepdim=True) + self.eps) * self.weights.float().unsqueeze(1)
        return y.sum(0) * self.coef


@dataclass
class PostNormed:
    """A pending delta that is normalised before it is added: x += value / rms(value) * weight, where ``value`` is a
    float32 tensor [T, H], a float32 stack [P, T, H] of partial sums, or a :class:`NormedSum`.  The norm that adds it
    (``Norm.forward``) does both in one pass."""

    value: object
    weight: torch.Tensor
    eps: float

    def resolve(self) -> torch.Tensor:
        v = self.value.resolve() if isinstance(self.value, NormedSum) else self.value.float()
        if v.dim() == 3:
            v = v.sum(0)
        return v * torch.rsqrt((v * v).mean(-1, keepdim=True) + self.eps) * self.weight.float()


@dataclass
class DepthAverage:
    """What a schedule entry with ``average`` hands on: the stream, once ``pending`` (a tensor, a stack of partial sums, a
    :class:`PostNormed`, or None) is added to it, is the entry's result X_index; what follows reads
    sum_{j < index} weights[j] history[j] + weights[index] X_index.  ``history`` float32 [> index, T, H] holds X_0 (the
    embedding output) and the earlier entries' results; the norm that forms the average stores X_index there too when a
    later entry needs it (``keep``).  ``rows``: the history's rows of the stream's rows, when the stream holds only some of
    the step's."""

    pending: object
    history: torch.Tensor
    weights: torch.Tensor
    index: int
    keep: bool = True
    rows: Optional[torch.Tensor] = None

    def resolve(self, residual: torch.Tensor) -> torch.Tensor:
        """The averaged stream itself, by library operations (traces and tests)."""
        p = self.pending
        if p is None or isinstance(p, StreamCopy):
            x = residual
        elif hasattr(p, "resolve"):
            x = residual + p.resolve()
        else:
            x = residual + (p.sum(0) if p.dim() == 3 else p.float())
        h = self.history[:self.index] if self.rows is None else self.history[:self.index, self.rows.long()]
        w = self.weights.float()
        return (w[:self.index, None, None] * h).sum(0) + w[self.index] * x


@dataclass
class StreamCopy:
    """What an arrangement hands on in the place of a pending delta when nothing is pending: the float32 stream is
    complete, and ``value`` is the same stream in the compute dtype, ready for the next matrix products (the stream
    itself when the compute dtype is float32).  Blocks that normalise after the sum read the stream itself, so the
    kernel that finishes a row also writes this copy."""

    value: torch.Tensor

    def resolve(self) -> int:
        return 0


# ------------------------------------------------------------------------------- parts
class Part:
    # False if ``forward`` waits for the device (reads a result on the host) or launches work whose
    # shape depends on data: a model with such a part is never replayed from a CUDA graph.
    capturable = True

    def __init__(self, runtime: Runtime):
        self.runtime = runtime

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        """Local tensor name -> what is expected of it."""
        return {}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Receive the loaded tensors (same local names); may fuse or re-lay them."""

    def shared_tensors(self) -> Tuple[str, ...]:
        """Full names of tensors of the MODEL (``ModelSpec.extra_tensors``) that this part reads besides its own: a
        table that all layers share.  The model hands them to ``bind_shared``."""
        return ()

    def bind_shared(self, tensors: Dict[str, torch.Tensor]) -> None:
        pass


class Mixer(Part):
    # Set by the model when every norm takes partial sums: the part may then return its output
    # as a float32 stack [splits, T, H] whose sum is the output (see Norm.accepts_partial_sums).
    partial_output = False

    # True if the part implements forward_tail.
    supports_tail = False

    # True if it implements forward_open_tail(x, step, cache, outs): forward_tail for blocks that take the output product
    # over (``forward_open``), leaving the wanted rows' activations in ``outs`` (nothing when there are no such rows).
    supports_open_tail = False

    def forward_tail(self, x: torch.Tensor, step: StepContext, cache) -> Optional[torch.Tensor]:
        """Update the cache (or state) for ALL rows of ``x`` as ``forward`` does, but return the
        output only for the rows ``step.tail_rows``, in that order (None when there are none);
        ``step.tail`` describes those rows as a step of their own."""
        raise NotImplementedError

    def cache_requirement(self):
        """PagedKV, FixedState, a tuple of those (a mixer made of several; its cache then has
        ``parts``), or None."""
        return None

    def forward(self, x: torch.Tensor, step: StepContext, cache: Optional[LayerCache]) -> torch.Tensor:
        raise NotImplementedError


class FeedForward(Part):
    partial_output = False   # as for Mixer

    def forward(self, x: torch.Tensor, step: StepContext) -> torch.Tensor:
        raise NotImplementedError


class Norm(Part):
    # True if ``delta`` may also be a float32 stack [splits, T, H] of partial sums, which the
    # norm adds in order before it adds them to the residual.
    accepts_partial_sums = False

    def forward(self, residual: torch.Tensor, delta: Optional[torch.Tensor],
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        raise NotImplementedError


class Embedder(Part):
    """Turns the step's token ids into the float32 stream when that takes more than a table row: ``forward(step,
    state, out, status, keep)`` fills ``out`` [T, width] (and ``keep``, when given, with the same rows) and returns a copy in
    the compute dtype (``out`` itself when that is float32) or None: nothing but the stream.  ``state_requirement()``: a :class:`FixedState` per request that the embedder keeps (for instance the last
    token of the request's previous step), or None.  Its tensors are named in full."""

    def state_requirement(self):
        return None

    def forward(self, step: StepContext, state: Optional[LayerCache], out: torch.Tensor, status: torch.Tensor,
                keep: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
        raise NotImplementedError


class Position(Part):
    """What the stock attention asks of an encoding that turns pairs (i, i + rotary_dim / 2) of a
    head's first ``rotary_dim`` elements: the attribute ``rotary_dim`` and ``cos_sin()``, a float32
    device table [positions, rotary_dim / 2, 2] of (cos, sin).  A mixer of another kind may ask its
    position part for anything else.

    ``pairs``: how the channels that turn together lie in a head, "halves" (i, i + rotary_dim / 2) or "neighbours"
    (2i, 2i + 1).  The kernels turn halves; ``halves_order`` is how a mixer serves neighbours with them."""

    pairs = "halves"

    def halves_order(self) -> List[int]:
        """The order of the first ``rotary_dim`` channels that makes the pairs halves: the old index of every new one.  A
        score does not depend on the order of the channels it is summed over, so a mixer may permute the rows of the
        projections in front of BOTH its sides by it, once, when the weights are loaded."""
        n = self.rotary_dim
        return list(range(n)) if self.pairs == "halves" else list(range(0, n, 2)) + list(range(1, n, 2))


def need_halves(position: Optional["Position"], what: str) -> None:
    """For mixers that hand their channels to the kernels as the checkpoint orders them."""
    if position is not None and getattr(position, "pairs", "halves") != "halves":
        raise ValueError(f"{what} turns pairs (i, i + rotary_dim / 2); an encoding of neighbouring channels is not built for it")


class Arrangement:
    """Wires the parts of one layer.  A subclass names its slots in ``SLOTS`` (slot name -> role:
    "mixer", "feed_forward" or "norm"; names in ``OPTIONAL`` may stay empty) and receives the
    built parts by slot name; each also becomes an attribute of that name (None when empty).
    ``forward`` takes and returns the pair (float32 residual stream, pending delta not yet added
    to it).  The model asks an arrangement only for what is below; it never names a slot."""

    SLOTS: Dict[str, str] = {}
    OPTIONAL: Tuple[str, ...] = ()

    def __init__(self, parts: Dict[str, Part]):
        unknown = sorted(set(parts) - set(self.SLOTS))
        missing = sorted(set(self.SLOTS) - set(parts) - set(self.OPTIONAL))
        if unknown or missing:
            raise ValueError(f"arrangement {type(self).__name__}: "
                             + (f"unknown slots {unknown} " if unknown else "")
                             + (f"missing slots {missing} " if missing else "")
                             + f"(slots: {sorted(self.SLOTS)})")
        self.slots = dict(parts)
        self.names: Optional[Dict[str, str]] = None     # LayerSpec.names, set by the model
        for name in self.SLOTS:
            setattr(self, name, parts.get(name))

    def parts(self) -> Dict[str, Part]:
        """Tensor-name component -> part (names follow the checkpoint)."""
        raise NotImplementedError

    def cache_owner(self) -> Optional[Part]:
        """The part whose ``cache_requirement`` decides what cache an execution of this layer
        gets (the first mixer by default), or None."""
        for name, role in self.SLOTS.items():
            if role == "mixer" and self.slots.get(name) is not None:
                return self.slots[name]
        return None

    def norms(self) -> List[Part]:
        return [self.slots[n] for n, role in self.SLOTS.items() if role == "norm" and n in self.slots]

    def producers(self) -> List[Part]:
        """The parts whose outputs go to a norm (mixers and feed-forwards)."""
        return [self.slots[n] for n, role in self.SLOTS.items() if role != "norm" and n in self.slots]

    def forward(self, residual, delta, step: StepContext, cache: Optional[LayerCache]):
        raise NotImplementedError

    # True if forward_tail may be called (the arrangement has one and its mixer can do it).
    supports_tail = False

    def forward_tail(self, residual, delta, step: StepContext, cache: Optional[LayerCache]):
        """As ``forward`` for the last entry of the schedule when ``step.tail`` is set: the
        returned pair holds only the rows ``step.tail_rows`` (or (None, None) without rows)."""
        raise NotImplementedError


MIXERS: Dict[str, type] = {}
FEED_FORWARDS: Dict[str, type] = {}
NORMS: Dict[str, type] = {}
POSITIONS: Dict[str, type] = {}
EMBEDDERS: Dict[str, type] = {}
ARRANGEMENTS: Dict[str, type] = {}


def _register(table: Dict[str, type], role: str, kind: str, cls: type, replace: bool) -> None:
    if not kind:
        raise ValueError(f"a {role} needs a non-empty kind")
    if kind in table and not replace:
        raise ValueError(f"{role} kind {kind!r} is already registered")
    table[kind] = cls


def register_mixer(kind, cls, replace=False): _register(MIXERS, "mixer", kind, cls, replace)
def register_feed_forward(kind, cls, replace=False): _register(FEED_FORWARDS, "feed_forward", kind, cls, replace)
def register_norm(kind, cls, replace=False): _register(NORMS, "norm", kind, cls, replace)
def register_position(kind, cls, replace=False): _register(POSITIONS, "position", kind, cls, replace)
def register_embedder(kind, cls, replace=False): _register(EMBEDDERS, "embedder", kind, cls, replace)
def register_arrangement(kind, cls, replace=False): _register(ARRANGEMENTS, "arrangement", kind, cls, replace)


def build_part(table: Dict[str, type], role: str, spec: PartSpec, runtime: Runtime, **extra):
    try:
        cls = table[spec.kind]
    except KeyError:
        raise ValueError(f"no {role} of kind {spec.kind!r} is registered "
                         f"(registered: {', '.join(sorted(table)) or 'none'})") from None
    return cls(runtime=runtime, **spec.params, **extra)
