"""Interfaces of the parts a layer is put together from.

A part is built from explicit sizes and constants (never from a model's configuration
object), states which tensors it wants (:meth:`Part.param_specs`, names relative to its own
prefix), receives them once (:meth:`Part.load`) and is then called by a block inside the step
function.  No part knows which model it is in.

=================  ==========================================================================
part               call
=================  ==========================================================================
Norm               ``forward(resid, delta, out_rows=None) -> normed``: add the pending
                   ``delta`` into the 32-bit residual stream, return norm(resid) in the compute
                   dtype; with ``out_rows`` only those rows are normed and resid is not written
PositionEncoding   ``apply(q, k, positions)`` in place on [N, heads, head_dim] views, or, for
                   the rotary encoding, its tables handed to the fused rotate-and-store kernel
Mixer              ``forward(x, batch, cache, write, position) -> [N, hidden]``; states what it
                   caches through ``kv_spec()`` (paged keys and values) and ``state_spec()``
                   (fixed-size state per request)
FeedForward        ``forward(x) -> [N, hidden]``
TokenEmbedding     ``embed(batch, table, resid, scale, state)``: the embedded tokens with something
                   beside their own vectors, into the stream
StreamJoin         ``forward(resid, first) -> resid``: the stream joined with the embedding
                   output, before a run that the model's run order marks
StreamMix          how a sublayer reads a stream of several parts and what its output does to them:
                   ``read`` (the reading weights) and ``update(output) -> pending``
Block              ``forward(resid, pending, batch, cache, write) -> pending``: the arrangement
                   of a layer's parts around the residual stream; its ``ROLES`` says which
                   parts it has (role -> kind of part), and it is built with one keyword
                   argument per role
=================  ==========================================================================
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import TYPE_CHECKING, Mapping

import torch

from ..weights.loader import ParamSpec

if TYPE_CHECKING:
    from ..engine.batch import StepBatch


@dataclass(frozen=True)
class BuildContext:
    """Where and in which precision a model is built.  ``dtype`` is the dtype of matrix-product
    operands and of the cache: ``torch.bfloat16`` (serving) or ``torch.float32`` (everything in
    true 32-bit)."""

    dtype: torch.dtype
    device: torch.device


@dataclass(frozen=True)
class KVSpec:
    """Paged keys and values one cache entry needs per token.  ``window`` None keeps every key;
    a number keeps the last ``window`` keys and lets older pages be given back.  ``planes`` 2: a
    page holds keys, then values; 1: one vector per token and kv head, which is its key and, by
    its leading entries, its value (a cache of latents)."""

    n_kv_heads: int
    head_dim: int
    window: int | None = None
    planes: int = 2


@dataclass(frozen=True)
class StateSpec:
    """State of fixed size that one cache entry keeps per live request."""

    shape: tuple[int, ...]
    dtype: torch.dtype


#: what a mixer's ``state_spec()`` may return: nothing, one tensor per request, or several
#: (``CacheView.state`` is then a tuple of tensors in the same order)
StateSpecs = StateSpec | tuple[StateSpec, ...] | None


@dataclass
class CacheView:
    """What one run of a layer sees of the cache in this step."""

    pages: torch.Tensor | None = None        # [n_pages, planes, n_kv_heads, page_size, head_dim]
    block_table: torch.Tensor | None = None  # int32 [rows, max_pages]; -1 where no page is held
    page_size: int = 0
    # [n_slots, *StateSpec.shape], or a tuple of such tensors for a mixer with several states
    state: torch.Tensor | tuple[torch.Tensor, ...] | None = None
    # the state of the layer's BLOCK for this cache entry (what the arrangement itself carries
    # from token to token, beside its mixer: a token shift's previous input), same forms
    block_state: torch.Tensor | tuple[torch.Tensor, ...] | None = None


class Part:
    #: False if ``forward`` reads device values on the host (``.item()``, ``.tolist()``) or
    #: otherwise cannot be recorded into a CUDA graph; decode steps are then launched plainly
    capturable = True
    #: True if the part takes a padded step: tokens after the last row's that belong to no row
    #: (``token_row`` -1, id 0, position 0; their activations are never read), rows without
    #: tokens, and counts in the batch that include them.  Small steps of any shape are then
    #: padded to a few sizes and replayed as CUDA graphs.  Parts that work on every token by
    #: itself are safe; the default is the careful one.
    pad_safe = False

    def param_specs(self) -> dict[str, ParamSpec]:
        return {}

    def load(self, tensors: Mapping[str, torch.Tensor], ctx: BuildContext) -> None:
        """Take the part's tensors (CPU or device, as stored) onto the device in the dtype the
        part computes in."""


class Norm(Part):
    def forward(self, resid: torch.Tensor, delta: torch.Tensor | None,
                out_rows: torch.Tensor | None = None) -> torch.Tensor:
        raise NotImplementedError

    def add_normed(self, resid: torch.Tensor, delta: torch.Tensor,
                   cast_out: torch.Tensor | None = None) -> None:
        """For layers that norm a branch's OUTPUT: ``resid += norm(delta)`` in 32-bit, and
        ``cast_out`` (if given) the updated stream in the compute dtype.  Optional."""
        raise NotImplementedError


class PositionEncoding(Part):
    #: True if the attention mixer may hand cos/sin tables to its fused rotate-and-store kernel
    rotary_tables = False

    def apply(self, q: torch.Tensor, k: torch.Tensor, positions: torch.Tensor) -> None:
        raise NotImplementedError


class Mixer(Part):
    def kv_spec(self) -> KVSpec | None:
        return None

    def state_spec(self) -> "StateSpecs":
        return None

    def forward(self, x: torch.Tensor, batch: "StepBatch", cache: CacheView, write: bool,
                position: PositionEncoding) -> torch.Tensor:
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


# Optional, for mixers and feed-forwards that END with a matrix product into the stream and sit
# in a block that joins its branches' output matrices into one product
# (:class:`scratch_llm_b200.parts.block.SharedNormBlock`):
#
#   out_segments() -> [(W [hidden, width], weight in the layer's sum), ...] | None   (after load)
#   activations_into(x, [batch, cache, write, position,] outs)   what each W multiplies, written
#       into the given column slices [N, width] of the block's buffer (a mixer takes the step's
#       arguments, a feed-forward x alone); in padded steps the slices hold zeros beforehand
#   release_out()   the part's own output matrices are no longer needed
#
# A mixer may also RETURN a weighted sum of tensors from forward()
# (:class:`scratch_llm_b200.parts.stream.Terms`) to a block and a norm that take one.


class TokenMix(Part):
    """Something that mixes a token's input with the previous token's before a mixer reads it
    (a token shift).  It states the state it carries (``state_spec()``) and offers what a norm
    that can do the mixing on its way needs; which norm kernels take it is the norm's word
    (``fuses_token_mix``)."""

    def state_spec(self) -> "StateSpecs":
        return None


class SideInput(Part):
    """Something a layer adds to the stream that depends on the step's tokens themselves (their
    ids, positions or rows) beside the stream: ``forward(x, batch) -> [N, hidden]``."""

    def forward(self, x: torch.Tensor, batch: "StepBatch") -> torch.Tensor:
        raise NotImplementedError


class TokenEmbedding(Part):
    """Something that the embedding adds to the tokens' own vectors (from their neighbours, for
    instance): ``embed`` fills the 32-bit stream with ``table[token] * scale`` plus its own
    contribution.  What it carries from token to token per live request it states in
    ``state_spec()`` and receives as ``state``."""

    def state_spec(self) -> "StateSpecs":
        return None

    def embed(self, batch: "StepBatch", table: torch.Tensor, resid: torch.Tensor, scale: float,
              state) -> None:
        raise NotImplementedError


class StreamJoin(Part):
    """Something that replaces the residual stream, between two runs of layers, by a function of
    the stream and of the embedding output (what the embedding left in the stream before the
    first layer): ``forward(resid, first) -> resid`` on 32-bit [N, hidden] tensors; the result
    may be a new tensor.  A model's run order says before which runs a join happens."""

    def forward(self, resid: torch.Tensor, first: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


class StreamMix(Part):
    """How a sublayer reads a residual stream of several parts (``ModelSpec.streams``; the stream
    is then [N, parts, hidden]) and what its output does to them: ``read`` (float32 [parts]) goes
    to the norm in front of the sublayer, ``update(output)`` is what the sublayer leaves pending
    (:class:`~.stream.StreamUpdate`), which the next norm carries out."""

    read: torch.Tensor | None = None

    def update(self, value):
        raise NotImplementedError


class Block:
    """An arrangement of a layer's parts.  ``ROLES`` maps each role the arrangement has onto
    the kind of part that fills it: ``"mixer"``, ``"feed_forward"``, ``"norm"`` or
    ``"position"``, ``"side"``, ``"token_mix"`` or ``"stream_mix"`` (the registry the part's spec is looked up in).  The model builds the parts
    from the layer's specs and constructs the block with one keyword argument per role.  At most
    one role may be a mixer: it owns the layer's cache entry."""

    ROLES: dict[str, str] = {}
    #: roles a layer may leave out (the block is then built without that keyword argument)
    OPTIONAL_ROLES: frozenset = frozenset()
    capturable = True
    pad_safe = False
    #: True if forward() takes ``next_entry=``: the (norm, part) that the next block in the run
    #: order starts with (None at the end), so that the block's last product may prepare it
    takes_next_entry = False

    def entry(self):
        """(norm, part) this block starts with, for the block before it; None: not said."""
        return None

    def state_spec(self) -> "StateSpecs":
        """State of fixed size that the arrangement itself keeps per live request and cache
        entry, beside its mixer's (``CacheView.block_state``); None: nothing."""
        return None

    def forward(self, resid: torch.Tensor, pending: torch.Tensor | None, batch: "StepBatch",
                cache: CacheView, write: bool) -> torch.Tensor:
        raise NotImplementedError
