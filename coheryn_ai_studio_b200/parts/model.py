"""The decoder as data: an embedding, layers built from a ModelSpec, a schedule that says
in which order (and how often, and with whose cache) they run, a final norm and the
output head.  It knows no architecture by name.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from .. import ops
from ..config.spec import ModelSpec
from ..weights.spec import TensorSpec
from . import attention, block, embedding, feedforward, norm, position, recurrent, routed  # noqa: F401  (register the stock parts)
from .base import (ARRANGEMENTS, EMBEDDERS, FEED_FORWARDS, MIXERS, NORMS, POSITIONS, DepthAverage, LayerCache, Part,
                   Runtime, StepContext, StreamCopy, build_part)


class DecoderModel:
    def __init__(self, spec: ModelSpec, runtime: Runtime):
        spec.validate()
        self.spec, self.runtime = spec, runtime
        self._positions: Dict[str, Part] = {}
        self.layers = []
        tables = {"mixer": MIXERS, "feed_forward": FEED_FORWARDS, "norm": NORMS}
        for ls in spec.layers:
            pos = None
            if ls.position is not None:
                key = repr(ls.position)
                if key not in self._positions:  # layers with the same encoding share its table
                    self._positions[key] = build_part(POSITIONS, "position", ls.position, runtime)
                pos = self._positions[key]
            try:
                arr = ARRANGEMENTS[ls.arrangement]
            except KeyError:
                raise ValueError(f"no arrangement {ls.arrangement!r} is registered") from None
            built = {}
            for slot, part_spec in ls.parts.items():
                role = arr.SLOTS.get(slot)
                if role is None:
                    raise ValueError(f"layer {ls.prefix}: arrangement {ls.arrangement!r} has no slot {slot!r} "
                                     f"(slots: {sorted(arr.SLOTS)})")
                extra = {"position": pos} if role == "mixer" and pos is not None else {}
                built[slot] = build_part(tables[role], role, part_spec, runtime, **extra)
            layer = arr(built, **dict(ls.arrangement_params))
            layer.names = dict(ls.names) if ls.names is not None else None
            self.layers.append(layer)
        self.final_norm = build_part(NORMS, "norm", spec.final_norm, runtime)
        self.embedder = build_part(EMBEDDERS, "embedder", spec.embedder, runtime) if spec.embedder is not None else None
        # Outputs go from a layer to the NEXT norm (the following layer's, or the final one),
        # so partial sums may flow only if every norm of the model can add them.
        norms = [n for layer in self.layers for n in layer.norms()] + [self.final_norm]
        if all(n.accepts_partial_sums for n in norms):
            for layer in self.layers:
                for part in layer.producers():
                    part.partial_output = True
        self.capturable = all(part.capturable for _, part in self._named_parts()) and all(
            p.capturable for p in self._positions.values()) and (self.embedder is None or self.embedder.capturable)
        self.embedding: Optional[torch.Tensor] = None
        self.head: Optional[torch.Tensor] = None
        self.head_bias: Optional[torch.Tensor] = None
        self.extra: Dict[str, torch.Tensor] = {}
        self.status = None
        # Called with (schedule entry, float32 [T, H] output of that entry) when set: the layer
        # outputs of a trace (crates/coheryn-engine/src/inference.rs:541-543).  Off in serving.
        self.layer_observer = None

    # ------------------------------------------------------------------ tensors
    def _named_parts(self) -> List[Tuple[str, Part]]:
        out = []
        for ls, layer in zip(self.spec.layers, self.layers):
            for comp, part in layer.parts().items():
                out.append((f"{ls.prefix}.{comp}", part))
        out.append((self.spec.final_norm_name, self.final_norm))
        return out

    @staticmethod
    def _join(prefix: str, local: str) -> str:
        return f"{prefix}.{local}" if local else prefix       # a part may name its one tensor as the part is named

    def _matrix_name(self, name: str) -> str:
        return name if self.spec.bare_tensor_names else f"{name}.weight"

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        """Every tensor the checkpoint must hold, by its full name."""
        s = self.spec
        if self.embedder is not None:
            specs = dict(self.embedder.tensor_specs())       # it owns the table and names its tensors in full
        else:
            specs = {self._matrix_name(s.embedding_name): TensorSpec((s.vocab_size, s.hidden_size))}
        for prefix, part in self._named_parts():
            for local, ts in part.tensor_specs().items():
                specs[self._join(prefix, local)] = ts
        if s.head_name is not None:
            specs[self._matrix_name(s.head_name)] = TensorSpec((s.vocab_size, s.hidden_size))
        if s.head_bias_name is not None:
            specs[s.head_bias_name] = TensorSpec((s.vocab_size,), role="vector", init="bias")
        for name, (shape, role, init) in s.extra_tensors.items():
            specs[name] = TensorSpec(tuple(shape), role=role, init=init)
        return specs

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        if self.embedder is not None:
            self.embedder.bind({name: tensors[name] for name in self.embedder.tensor_specs() if name in tensors})
        self.embedding = tensors.get(self._matrix_name(s.embedding_name))
        if self.embedding is None and (self.embedder is None or s.head_name is None):
            raise KeyError(self._matrix_name(s.embedding_name))
        for prefix, part in self._named_parts():
            local = {name: tensors[self._join(prefix, name)] for name in part.tensor_specs()
                     if self._join(prefix, name) in tensors}
            part.bind(local)
            shared = part.shared_tensors()
            if shared:
                part.bind_shared({name: tensors[name] for name in shared})
        self.head = tensors[self._matrix_name(s.head_name)] if s.head_name is not None else self.embedding
        self.head_bias = tensors[s.head_bias_name] if s.head_bias_name is not None else None
        self.extra = {name: tensors[name] for name in s.extra_tensors}
        for e in s.schedule:      # what enters the residual sum is float32
            if e.average is not None:
                self.extra[e.average] = self.extra[e.average].to(torch.float32).contiguous()
        self.status = torch.zeros(1, dtype=torch.int32, device=self.runtime.device)

    # ------------------------------------------------------------------ cache needs
    def cache_requirements(self):
        """Per schedule entry: the mixer's requirement, or None when the entry reads an
        earlier entry's cache."""
        def need(entry):
            owner = self.layers[entry.layer].cache_owner()
            return owner.cache_requirement() if owner is not None and entry.cache_from is None else None
        needs = [need(e) for e in self.spec.schedule]
        # what the model itself keeps per request follows the schedule's entries
        if self.embedder is not None and self.embedder.state_requirement() is not None:
            needs.append(self.embedder.state_requirement())
        return needs

    # ------------------------------------------------------------------ forward
    def forward(self, step: StepContext, caches: List[Optional[LayerCache]],
                logit_rows: torch.Tensor) -> torch.Tensor:
        """Run the step's tokens through the schedule; return float32 logits
        ``[len(logit_rows), vocab]`` of the rows asked for."""
        T, H = step.num_tokens, self.spec.hidden_size
        step.native = None      # a step object may be run again (warm-up, then capture): on another stream
        step.shared = {}
        residual = torch.empty((T, H), dtype=torch.float32, device=self.runtime.device)
        delta = None
        last = len(self.spec.schedule) - 1
        # the results that averages over depth read: the embedding output, then every entry's that a later average needs
        averaged = [i for i, e in enumerate(self.spec.schedule) if e.average is not None]
        history = None
        if averaged:
            history = torch.empty((averaged[-1] + 1, T, H), dtype=torch.float32, device=self.runtime.device)
        keep = history[0] if history is not None else None
        if self.embedder is not None:
            own = caches[len(self.spec.schedule)] if len(caches) > len(self.spec.schedule) else None
            copy = self.embedder.forward(step, own, residual, self.status, keep)
            delta = StreamCopy(copy) if copy is not None else None
        else:
            ops.embed_gather(self.embedding, step.token_ids, residual, self.status, scale=self.spec.embedding_scale, copy=keep)
        tailed = False
        for i, (entry, cache) in enumerate(zip(self.spec.schedule, caches)):
            layer = self.layers[entry.layer]
            if entry.inject is not None and isinstance(delta, DepthAverage):
                norm.apply_depth_average(residual, delta, None, 0.0, None)      # the stream itself, nothing pending
                delta = None
            if entry.inject is not None and entry.inject.mix is not None:
                # the stream, with what is pending, beside the embedding output: one kernel makes the product's input,
                # the product's float32 result is the new stream and nothing is pending
                if delta is not None and not isinstance(delta, torch.Tensor):
                    pending = delta.resolve()
                    delta = None if isinstance(pending, int) else pending
                joined = ops.stream_join(residual, delta, self.embedding, step.token_ids, self.spec.embedding_scale,
                                         self.runtime.dtype)
                residual = ops.linear(joined, self.extra[entry.inject.mix], out_dtype=torch.float32)
                delta = None
            elif entry.inject is not None:
                # added to the stream itself; what the previous entry handed on stays pending beside it
                vec = entry.inject.vector
                ops.stream_inject(residual, self.embedding if entry.inject.embedding else None, step.token_ids,
                                  self.spec.embedding_scale, self.extra[vec[0]][vec[1]] if vec is not None else None)
            if i == last and step.tail is not None and layer.supports_tail and self.layer_observer is None:
                residual, delta = layer.forward_tail(residual, delta, step, cache)
                tailed = True
            else:
                residual, delta = layer.forward(residual, delta, step, cache)
            if history is not None and residual is not None and i <= averaged[-1]:
                delta = DepthAverage(None if isinstance(delta, StreamCopy) else delta, history, self.extra[entry.average], i + 1,
                                     keep=i < averaged[-1], rows=step.tail_rows if tailed else None)
            if self.layer_observer is not None:
                if delta is None or isinstance(delta, StreamCopy):
                    out = residual
                elif isinstance(delta, DepthAverage):
                    out = delta.resolve(residual)
                elif hasattr(delta, "resolve"):      # a summand that is normalised before it is added
                    out = residual + delta.resolve()
                else:
                    out = residual + (delta.sum(0) if delta.dim() == 3 else delta.float())
                self.layer_observer(i, out)
        R = logit_rows.numel()
        if R == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=self.runtime.device)
        if isinstance(delta, StreamCopy):       # nothing is pending
            delta = None
        h = self.final_norm.forward(residual, delta, rows=None if tailed else logit_rows)
        logits = ops.linear(h, self.head, out_dtype=torch.float32)
        if self.spec.logit_scale is not None or self.head_bias is not None or self.spec.logit_softcap is not None:
            ops.scale_add_bias(logits, self.spec.logit_scale, self.head_bias, self.spec.logit_softcap)
        return logits
