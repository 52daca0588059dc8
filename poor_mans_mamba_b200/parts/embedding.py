"""Rows that join the embedding's row of a token.

``bigram``: a second table whose row depends on the token before, too,

    x_t = E[token_t] + B[(token_(t-1) * mul_prev + token_t * mul_cur) mod buckets],      B [buckets + 1, D];

a sequence's first token takes the last row of B.  State per request: the last token plus one (an integer in a
slot; zero: there is none yet).  The row
is added in the embedding's launch; the block of a sequence's first token of the step reads the state and then
leaves the step's last token there.
"""
from __future__ import annotations

from typing import Any, Dict, List

import torch

from .base import EmbeddingAddend, ParamSpec, StateSpec, register_embedding_addend

Tensor = torch.Tensor


class BigramEmbedding(EmbeddingAddend):
    def __init__(self, hidden_size: int, buckets: int, mul_prev: int, mul_cur: int, tensor: str = ""):
        if buckets < 1 or mul_prev < 0 or mul_cur < 0:
            raise ValueError("at least one bucket, multipliers that are not negative")
        self.hidden_size, self.buckets = int(hidden_size), int(buckets)
        self.mul_prev, self.mul_cur, self.tensor = int(mul_prev), int(mul_cur), str(tensor)

    def param_specs(self) -> List[ParamSpec]:
        return [ParamSpec(self.tensor, (self.buckets + 1, self.hidden_size))]

    def state_specs(self) -> List[StateSpec]:
        return [StateSpec.fixed("previous", (1,), "int32")]

    def bind(self, params: Dict[str, Tensor]) -> None:
        self.table = params[self.tensor].contiguous()

    def arguments(self, ctx, cache) -> Dict[str, Any]:
        return {"bigram": (self.table, self.mul_prev, self.mul_cur), "previous": cache.fixed(f"{self.name}.previous"),
                "seq_of": ctx.seq_of, "cu": ctx.cu_seqlens, "slots": ctx.slots}


register_embedding_addend("bigram", BigramEmbedding)
