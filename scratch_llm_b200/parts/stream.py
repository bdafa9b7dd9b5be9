"""Handing a branch's output to the next norm without a kernel of its own, in decode steps.

In a pre-norm layer a branch ends with a matrix product whose output is added to the residual
stream, a norm follows, and the next branch starts with a matrix product
(src/scratch_llm/model.py:423-436 of the reference: ``x + Attn(Norm(x))``, ``x + FFN(Norm(x))``).
With a handful of tokens each of these is a short kernel and the step's time is the chain of
their starts and ends.  Two of the kernels can go, because an RMS norm's factor
``rsqrt(mean(x^2) + eps)`` is ONE number per token and commutes with the product that follows:

* the product that ends a branch (:class:`StreamSink`) adds its output into the 32-bit stream
  itself, writes ``stream * gain`` in the compute dtype as the next product's input, and leaves
  each token's sum of squares in shares (one per 8 features);
* the product that starts the next branch takes that input as it is (:class:`Normed`) and
  multiplies its outputs by the token's factor, which it gets by adding the shares in a fixed
  order.

The norm's arithmetic stays 32-bit with one rounding of the activations; only the place of
that rounding moves (before the factor instead of after it).  Parts opt in: a mixer or
feed-forward that can end with a sink takes a ``sink`` argument and says ``accepts_sink``; one
that can start from unfinished activations says so through ``accepts_normed(n_tokens)``; a norm
whose factor is one number per token says ``deferrable``.  Everything else runs as before.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ..kernels import ops


@dataclass
class Normed:
    """Activations whose norm is not finished: the true value of row t is
    ``x[t] * rsqrt(shares[:, t].sum() / dim + eps)``."""

    x: torch.Tensor          # [tokens, dim] in the compute dtype: stream * gain
    shares: torch.Tensor     # float32 [parts, 8]: sums of squares of the stream, per token
    dim: int
    eps: float
    norm: object             # the norm this stands for

    @property
    def shape(self):
        return self.x.shape


@dataclass
class Current:
    """Nothing is pending: the stream is up to date, and ``x`` is its copy in the compute dtype
    (the stream itself where that dtype is 32-bit), for a block whose branches read the stream
    as it is.  A norm that meets it adds nothing."""

    x: torch.Tensor


@dataclass
class RoutedSum:
    """A routed feed-forward's output that is not added up yet: token n's is ``sum_j weights[n, j]
    * y[place[n, j]]`` over its choices, plus ``sigmoid(gate[n]) * shared[n]`` (without ``gate``:
    plus ``shared[n]``; without ``shared``: nothing).  A norm that takes it (``takes_routed``)
    adds it up in 32-bit while it reads the stream."""

    y: torch.Tensor               # float32 [places, hidden]
    ids: torch.Tensor             # int32 [tokens, top]
    weights: torch.Tensor         # float32 [tokens, top]
    place: torch.Tensor           # int32 [tokens * top], -1: no row
    shared: torch.Tensor | None   # [tokens, hidden] in the compute dtype
    gate: torch.Tensor | None     # float32 [tokens, 1]


@dataclass
class Terms:
    """What a layer leaves pending for the stream when it is a weighted sum of several branch
    outputs: the stream is to receive ``sum(coef * tensor)``, plus a routed feed-forward's
    output (``routed``, weight 1) where the norm takes one.  A norm that takes it
    (``takes_terms``) forms the sum in 32-bit while it reads the stream, so that neither the
    sum nor the products by the weights cost a pass or a rounding of their own."""

    items: tuple            # ((tensor [tokens, hidden], coefficient), ...)
    routed: RoutedSum | None = None

    def scaled(self, factor: float) -> "Terms":
        if self.routed is not None and factor != 1.0:
            raise ValueError("a routed sum has no weight of its own")
        return Terms(tuple((t, c * factor) for t, c in self.items), self.routed)

    @staticmethod
    def of(value, coef: float = 1.0) -> "Terms":
        """``coef * value`` as terms, whether ``value`` is a tensor or already a sum."""
        if isinstance(value, RoutedSum):
            return Terms((), value).scaled(coef)
        if isinstance(value, Terms):
            return value.scaled(coef)
        return Terms(((value, float(coef)),))

    def __add__(self, other: "Terms") -> "Terms":
        if self.routed is not None and other.routed is not None:
            raise ValueError("a sum takes one routed output")
        return Terms(self.items + other.items, self.routed or other.routed)

    def total(self) -> torch.Tensor:
        """The sum as a 32-bit tensor, for looking into a model."""
        out = sum(c * t.float() for t, c in self.items)
        r = self.routed
        if r is not None:
            n, top = r.ids.shape
            place = r.place.view(n, top).long()
            rows = r.y[place.clamp(min=0)] * (place >= 0)[..., None]
            out = out + (r.weights[..., None] * rows).sum(1)
            if r.shared is not None:
                out = out + r.shared.float() * (torch.sigmoid(r.gate) if r.gate is not None else 1.0)
        return out


@dataclass
class StreamUpdate:
    """What a sublayer leaves pending for a residual stream of several parts [tokens, parts, hidden]:
    ``x_t <- sum_s mix[s, t] x_s + to[t] * y`` with y the sum of ``terms``.  A norm that says
    ``takes_streams`` carries it out while it reads the parts for the next sublayer."""

    terms: Terms
    mix: torch.Tensor     # float32 [parts, parts], [from, to]
    to: torch.Tensor      # float32 [parts]

    def applied(self, parts: torch.Tensor) -> torch.Tensor:
        """The updated parts as a new tensor, for looking into a model."""
        y = self.terms.total()
        return torch.einsum("nsd,st->ntd", parts, self.mix) + self.to[None, :, None] * y[:, None]


class StreamSink:
    """Where a branch's last product may put its output: into ``resid``, prepared for ``norm``."""

    #: steps of more tokens never hand a norm over (the kernels that can are small-batch ones)
    MAX_TOKENS = 8

    def __init__(self, resid: torch.Tensor, norm) -> None:
        self.resid, self.norm = resid, norm

    def finish(self, linear, x: torch.Tensor):
        """``linear(x)`` added into the stream: a :class:`Normed` for the norm that follows, or,
        where the product's kernel cannot do that, the plain output (the norm then runs as
        usual)."""
        if not linear.can_sink(x):
            return linear(x)
        n, d = x.shape[0], linear.out_features
        x_out = torch.empty((n, d), dtype=x.dtype, device=x.device)
        shares = torch.empty((-(-d // 8), 8), dtype=torch.float32, device=x.device)
        ops.gemv_tma(x, linear.weight, None,
                     sink=(self.resid, self.norm.weight, x_out, shares))
        return Normed(x_out, shares, d, self.norm.eps, self.norm)
