"""Embedders: what turns token ids into the stream when a table row is not all of it.

``pair_hash_embedding``: x_t = table[id_t] (* scale) + pair[(id_{t-1} * mul_prev + id_t * mul_cur) mod buckets], with
row ``buckets`` of ``pair`` (its last) for the first token of a sequence, then optionally x / rms(x) * (norm + offset).
Without pair rows it is a table row with a norm behind it.  The token
before the first one of a step's portion is the last token of the request's previous step: one int32 word of fixed state
per request, written by the same step after it was read.  One kernel makes the float32 stream and its copy in the
compute dtype.

``position_table_embedding``: x_t = table[id_t] (* scale) + positions[p_t], a learned row per position.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import ops
from ..weights.spec import TensorSpec
from .base import Embedder, FixedState, LayerCache, Runtime, StepContext, register_embedder


class PairHashEmbedding(Embedder):
    def __init__(self, runtime: Runtime, vocab_size: int, hidden_size: int, table: str, pair: Optional[str] = None,
                 buckets: int = 0, mul_prev: int = 0, mul_cur: int = 0, norm: Optional[str] = None, eps: float = 1e-6,
                 scale: Optional[float] = None, norm_offset: float = 0.0, compute_copy: bool = True):
        """``table``, ``pair``, ``norm``: full tensor names ([vocab, width], [buckets + 1, width], [width]); ``pair`` None:
        no pair rows; ``norm`` None: no norm.  ``norm_offset``: what is added to the stored norm weight (1 for weights that are
        stored around zero).  ``compute_copy`` False: nothing but the float32 stream (for blocks that normalise it first)."""
        super().__init__(runtime)
        self.vocab_size, self.hidden_size = int(vocab_size), int(hidden_size)
        self.table_name, self.pair_name, self.norm_name = str(table), pair, norm
        self.buckets, self.mul_prev, self.mul_cur = int(buckets), int(mul_prev), int(mul_cur)
        if pair is not None and (self.buckets < 1 or self.mul_prev < 0 or self.mul_cur < 0):
            raise ValueError("pair rows need a positive number of buckets and non-negative multipliers")
        self.eps, self.scale, self.norm_offset, self.compute_copy = float(eps), scale, float(norm_offset), bool(compute_copy)
        self.table = self.pair = self.norm = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        specs = {self.table_name: TensorSpec((self.vocab_size, self.hidden_size))}
        if self.pair_name is not None:
            specs[self.pair_name] = TensorSpec((self.buckets + 1, self.hidden_size))
        if self.norm_name is not None:
            specs[self.norm_name] = TensorSpec((self.hidden_size,), role="vector", init="norm" if self.norm_offset == 0.0 else "centered")
        return specs

    def bind(self, tensors):
        self.table = tensors[self.table_name]
        self.pair = tensors[self.pair_name] if self.pair_name is not None else None
        self.norm = tensors[self.norm_name] if self.norm_name is not None else None
        if self.norm is not None and self.norm_offset != 0.0:
            self.norm = (self.norm.to(torch.float64) + self.norm_offset).to(torch.float32).contiguous()

    def state_requirement(self):
        return FixedState((1,), torch.int32) if self.pair_name is not None else None

    def forward(self, step: StepContext, state: Optional[LayerCache], out: torch.Tensor, status: torch.Tensor,
                keep: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
        if keep is not None:
            raise ValueError("pair_hash_embedding: a second copy of the embedding output is not built")
        cast = None
        if self.compute_copy:
            cast = out if self.runtime.dtype == torch.float32 else torch.empty(out.shape, dtype=self.runtime.dtype, device=out.device)
        last = state.state if state is not None else None
        ops.embed_pair(self.table, self.pair, step, last, self.mul_prev, self.mul_cur, self.buckets, self.scale, self.norm,
                       self.eps, out, None if cast is out else cast, status)
        if last is not None:
            ops.store_last_ids(step, last)
        return cast


class PositionTableEmbedding(Embedder):
    def __init__(self, runtime: Runtime, vocab_size: int, hidden_size: int, table: str, positions: str, max_positions: int,
                 scale: Optional[float] = None):
        """``table``, ``positions``: full tensor names ([vocab, width], [max_positions, width])."""
        super().__init__(runtime)
        self.vocab_size, self.hidden_size, self.max_positions = int(vocab_size), int(hidden_size), int(max_positions)
        self.table_name, self.positions_name, self.scale = str(table), str(positions), scale
        self.table = self.rows = None

    def tensor_specs(self) -> Dict[str, TensorSpec]:
        return {self.table_name: TensorSpec((self.vocab_size, self.hidden_size)),
                self.positions_name: TensorSpec((self.max_positions, self.hidden_size))}

    def bind(self, tensors):
        self.table, self.rows = tensors[self.table_name], tensors[self.positions_name]

    def forward(self, step: StepContext, state: Optional[LayerCache], out: torch.Tensor, status: torch.Tensor,
                keep: Optional[torch.Tensor] = None) -> None:
        ops.embed_gather(self.table, step.token_ids, out, status, scale=self.scale, pos_table=self.rows, positions=step.positions,
                         copy=keep)


register_embedder("position_table_embedding", PositionTableEmbedding)
register_embedder("pair_hash_embedding", PairHashEmbedding)
