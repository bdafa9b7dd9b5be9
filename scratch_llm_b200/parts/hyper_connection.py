"""Hyper-connections: a residual stream of several parts ``x_1 .. x_s`` (all equal to the embedding
output at the start) instead of one sum.  In front of a sublayer

    u = sum_s in[s] x_s,      y = sublayer(norm(u))

and after it every part from all old ones at once,

    x_t <- sum_s mix[s, t] x_s + residual_mult * out[t] * y          (mix is indexed [from, to])

with the small learned tensors ``in`` [s], ``out`` [s] and ``mix`` [s, s] of that sublayer.  The model's
output is the sum of the parts.  ``learned=False``: no tensors, the weights are 1 and ``mix`` is the
identity; with one part that is the plain residual sum with a multiplier.

Nothing is computed here: the block hands a sublayer's output on as a :class:`~.stream.StreamUpdate`,
and the next norm (one that says ``takes_streams``) forms the update, the reading and the norm in one
pass.
"""

from __future__ import annotations

from typing import Mapping

import torch

from ..kernels import ops
from ..weights.loader import ParamSpec
from .base import BuildContext, StreamMix
from .registry import register_stream_mix
from .stream import StreamUpdate, Terms


@register_stream_mix("hyper_connection")
class HyperConnection(StreamMix):
    pad_safe = True   # every token by itself

    def __init__(self, streams: int, residual_mult: float = 1.0, learned: bool = True,
                 names: Mapping[str, str] | None = None) -> None:
        if not 1 <= streams <= ops.STREAMS_MAX:
            raise ValueError(f"streams must be 1 to {ops.STREAMS_MAX}, got {streams}")
        self.streams, self.residual_mult = streams, float(residual_mult)
        self.learned = bool(learned)
        self.names = {"in": "in", "out": "out", "mix": "mix", **(names or {})}
        self.read = self.to = self.mix = None

    def kernel_jobs(self, dtype: torch.dtype):
        return [ops.core_job("sllm_streams")]

    def param_specs(self) -> dict[str, ParamSpec]:
        if not self.learned:
            return {}
        s, n = self.streams, self.names
        return {n["in"]: ParamSpec((s,), "gain"), n["out"]: ParamSpec((s,), "gain"),
                n["mix"]: ParamSpec((s, s), "gain")}

    def load(self, tensors: Mapping[str, torch.Tensor], ctx: BuildContext) -> None:
        put = lambda t: t.to(device=ctx.device, dtype=torch.float32).contiguous()  # noqa: E731
        if self.learned:
            read, out, mix = (tensors[self.names[k]] for k in ("in", "out", "mix"))
        else:
            read, out, mix = torch.ones(self.streams), torch.ones(self.streams), \
                torch.eye(self.streams)
        self.read, self.mix = put(read), put(mix)
        self.to = put(out) * self.residual_mult

    def update(self, value) -> StreamUpdate:
        """A sublayer's output (a tensor, Terms or a RoutedSum) as what is pending for the parts."""
        return StreamUpdate(Terms.of(value), self.mix, self.to)
