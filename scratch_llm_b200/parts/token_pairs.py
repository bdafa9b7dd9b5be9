"""An embedding for the pair (previous token, token), added to the token's own embedding:

    x = embed[token] + table[(previous * mul_prev + token * mul_cur) mod buckets]

and, for a sequence's first token, the table's last row, number ``buckets``.  The previous token
is state: each request's last token is carried from step to step in its state slot (on the
device, where a token that a sampler has just chosen is known before the host has read it).
"""

from __future__ import annotations

from typing import Mapping

import torch

from ..kernels import ops
from ..weights.loader import ParamSpec
from .base import BuildContext, StateSpec, TokenEmbedding
from .registry import register_token_embedding


@register_token_embedding("hashed_pairs")
class HashedPairs(TokenEmbedding):
    pad_safe = True   # padding tokens belong to no row: they read and leave no previous token

    def __init__(self, size: int, buckets: int, mul_prev: int, mul_cur: int) -> None:
        if buckets < 1 or mul_prev < 0 or mul_cur < 0:
            raise ValueError("hashed pairs: buckets must be positive, the multipliers not negative")
        self.size, self.buckets = size, buckets
        self.mul_prev, self.mul_cur = mul_prev, mul_cur
        self.table: torch.Tensor | None = None

    def state_spec(self) -> StateSpec:
        return StateSpec((), torch.int32)      # the last token

    def kernel_jobs(self, dtype: torch.dtype):
        return [ops.core_job("sllm_sum_norm")]

    def param_specs(self) -> dict[str, ParamSpec]:
        return {"": ParamSpec((self.buckets + 1, self.size))}

    def load(self, tensors: Mapping[str, torch.Tensor], ctx: BuildContext) -> None:
        self.table = tensors[""].to(device=ctx.device, dtype=ctx.dtype).contiguous()

    def embed(self, batch, table: torch.Tensor, resid: torch.Tensor, scale: float, state) -> None:
        ops.embed_pair(batch.token_ids, batch.positions, batch.token_row, batch.row_start,
                       batch.row_slot, table, self.table, state, self.mul_prev, self.mul_cur,
                       resid, pending=batch.pending_tokens, scale=scale)
