"""A token's embedding plus the embedding of the pair it forms with the token before it.

    x_t = E[token_t] + P[(token_{t-1} * mul_prev + token_t * mul_cur) mod buckets],   x_0 = E[token_0] + P[buckets]

P has buckets + 1 rows, the last one for a sequence's first token.  The sum opens a float residual stream (it is never
rounded to 16 bits).  The token before a portion is part of a request's state: one integer in the cache manager's state slots.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import kernels
from ..weights.loader import TensorSpec
from .base import Embedding, StateSpec, register_part


class PairEmbedding(Embedding):
    graph_safe = True

    def __init__(self, vocab_size: int, size: int, table_name: str, pair_name: Optional[str] = None, buckets: int = 0,
                 mul_prev: int = 0, mul_cur: int = 0, **_):
        """`pair_name` None: the token's own row is the whole embedding."""
        self.V, self.size, self.n_table, self.n_pairs = int(vocab_size), int(size), table_name, pair_name
        self.buckets, self.mul_prev, self.mul_cur = int(buckets), int(mul_prev), int(mul_cur)
        if pair_name is not None and self.buckets <= 0:
            raise ValueError(f"a pair embedding needs a positive number of buckets, not {buckets}")
        self.table = self.pairs = None

    def tensor_specs(self) -> List[TensorSpec]:
        specs = [TensorSpec(self.n_table, (self.V, self.size), "embedding")]
        if self.n_pairs is not None:
            specs.append(TensorSpec(self.n_pairs, (self.buckets + 1, self.size), "embedding"))
        return specs

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.table = tensors[self.n_table].contiguous()
        self.pairs = tensors[self.n_pairs].contiguous() if self.n_pairs is not None else None

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((1,), torch.int32) if self.n_pairs is not None else None

    def open(self, ctx, state):
        T = ctx.launch_tokens
        stream = ctx.ws.get("residual_stream", T, self.size, torch.float32)
        kernels.pair_embedding(self.table, self.pairs, ctx.token_ids, ctx.positions, ctx.token_req, ctx.cu_q, ctx.state_slots, state,
                               stream, T, self.buckets, self.mul_prev, self.mul_cur, ctx.err)
        # nothing is pending on a stream that begins (a context may be walked twice)
        ctx.pending_norm = ctx.stream_keep = None
        return None, stream


register_part("embedding", "pair_embedding", PairEmbedding)
