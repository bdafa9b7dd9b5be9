"""Linear attention with decays: recurrent layers whose state per request is one matrix ``S`` [key,
value] per head in 32-bit.

``gated_linear_attention``: one decay per key channel, from the input through a low-rank pair,

    q = W_q h * key_dim^(-1/2),  k = W_k h  (H x key_dim),   v = W_v h  (H x value_dim)
    alpha = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)                           laid out H x key_dim
    S <- diag(alpha) S + k v^T,   o = S^T q
    out = W_o ( rmsnorm_per_head(o) * gain * silu(W_g h) )     (gain: value_dim entries, every head's)

``lightning_attention``: one constant decay per head,

    q = silu(W_q h),  k = silu(W_k h)  (H x key_dim),   v = silu(W_v h)  (H x value_dim)
    S <- decay_h S + k v^T,   o = S^T q
    out = W_o ( rmsnorm(all heads of o together) * gain * sigmoid(W_g h) )     (gain: H x value_dim)

The projections (with their silu) run in the compute dtype; the low-rank hidden values, everything of
the decays, the state and the read-out are 32-bit.  The state lives in the cache manager's state
slots, so a request may be fed in portions of any size, beside other requests, and its slot is used
again after it ends.
"""

from __future__ import annotations

import math
from typing import Mapping, Sequence

import torch

from ..kernels import ops
from ..weights.loader import ParamSpec
from .base import BuildContext, CacheView, Mixer, PositionEncoding, StateSpec
from .linear import Linear
from .registry import register_mixer


def stacked(blocks: Sequence[torch.Tensor]) -> tuple[Linear, list[int]]:
    """One product for several matrices of the same input, each starting on a 16-byte boundary of
    the output (zero rows in between): (the product, where each matrix's columns start)."""
    rows, cols, at = [], [], 0
    for w in blocks:
        cols.append(at)
        rows += [w, w.new_zeros((-w.shape[0] % 8, w.shape[1]))]
        at += -(-w.shape[0] // 8) * 8
    return Linear(torch.cat(rows, 0).contiguous()), cols


class _LinearAttention(Mixer):
    pad_safe = True   # padding tokens belong to no row: the recurrence never sees them

    def __init__(self, hidden_size: int, n_heads: int, key_dim: int, value_dim: int, eps: float,
                 names: Mapping[str, str] | None) -> None:
        if min(n_heads, value_dim) < 1:
            raise ValueError("linear attention: sizes must be positive")
        if not 1 <= key_dim <= ops.GATED_SCAN_MAX_KEY_DIM:
            raise ValueError(f"key size {key_dim}: the scan kernel takes 1 to "
                             f"{ops.GATED_SCAN_MAX_KEY_DIM}")
        self.hidden_size, self.n_heads = hidden_size, n_heads
        self.key_dim, self.value_dim, self.eps = key_dim, value_dim, float(eps)
        self.names = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm",
                      **(names or {})}
        self.proj: Linear | None = None      # [q; k; v; g]
        self.cols: list[int] = []            # where they start
        self.o: Linear | None = None
        self.gain = None

    @property
    def widths(self) -> tuple[int, int, int, int]:
        hk, hv = self.n_heads * self.key_dim, self.n_heads * self.value_dim
        return hk, hk, hv, hv

    def state_spec(self) -> StateSpec:
        return StateSpec((self.n_heads, self.value_dim, self.key_dim), torch.float32)

    def param_specs(self) -> dict[str, ParamSpec]:
        d, n = self.hidden_size, self.names
        specs = {n[c]: ParamSpec((w, d)) for c, w in zip("qkvg", self.widths)}
        specs[n["o"]] = ParamSpec((d, self.n_heads * self.value_dim))
        return specs

    def load(self, tensors: Mapping[str, torch.Tensor], ctx: BuildContext) -> None:
        put = lambda t: t.to(device=ctx.device, dtype=ctx.dtype)  # noqa: E731
        self.proj, self.cols = stacked([put(tensors[self.names[c]]) for c in "qkvg"])
        self.o = Linear(put(tensors[self.names["o"]]).contiguous())
        self.gain = tensors[self.names["norm"]].to(device=ctx.device,
                                                   dtype=torch.float32).contiguous()

    def _read_out_buffer(self, x, batch) -> torch.Tensor:
        # (padding tokens belong to no row: their read-out stays zero)
        return (torch.zeros if batch.padded else torch.empty)(
            (x.shape[0], self.n_heads * self.value_dim), dtype=torch.float32, device=x.device)

    def forward(self, x, batch, cache: CacheView, write: bool, position: PositionEncoding):
        if not write:
            raise NotImplementedError("a run that only reads another run's recurrent state")
        proj = self.proj(x)
        out = torch.empty((x.shape[0], self.widths[3]), dtype=proj.dtype, device=proj.device)
        self._mix(x, proj, batch, cache.state, self._read_out_buffer(x, batch), out)
        return self.o(out)

    def _split(self, proj: torch.Tensor):
        return [proj[:, c:c + w] for c, w in zip(self.cols, self.widths)]

    def _mix(self, x, proj, batch, state, o, out) -> None:
        """The recurrence's read-out, normed and gated, from ``proj`` (and x) into ``out``; ``o``: a
        32-bit buffer for the read-out."""
        raise NotImplementedError


@register_mixer("gated_linear_attention")
class GatedLinearAttention(_LinearAttention):
    def __init__(self, hidden_size: int, n_heads: int, key_dim: int, value_dim: int, tau: float,
                 eps: float, decay_rank: int = -1, names: Mapping[str, str] | None = None) -> None:
        """``decay_rank``: the low rank of the decay's pair of matrices (-1: as the tensors say)."""
        super().__init__(hidden_size, n_heads, key_dim, value_dim, eps,
                         {"a1": "a1", "a2": "a2", "a2_bias": "a2.b", **(names or {})})
        if not (tau > 0 and math.isfinite(tau)):
            raise ValueError(f"tau must be positive, got {tau!r}")
        self.tau, self.rank = float(tau), decay_rank
        self.a1: Linear | None = None        # 32-bit output
        self.a2t = self.a2_bias = None

    def kernel_jobs(self, dtype: torch.dtype):
        return [ops.core_job("sllm_recurrent_ops"), ops.core_job("sllm_channel_scan")]

    def param_specs(self) -> dict[str, ParamSpec]:
        n, hk = self.names, self.n_heads * self.key_dim
        return {**super().param_specs(), n["norm"]: ParamSpec((self.value_dim,), "gain"),
                n["a1"]: ParamSpec((self.rank, self.hidden_size)),
                n["a2"]: ParamSpec((hk, self.rank)), n["a2_bias"]: ParamSpec((hk,), "gain")}

    def load(self, tensors: Mapping[str, torch.Tensor], ctx: BuildContext) -> None:
        super().load(tensors, ctx)
        f32 = lambda t: t.to(device=ctx.device, dtype=torch.float32)  # noqa: E731
        a1, a2 = (tensors[self.names[n]] for n in ("a1", "a2"))
        if a1.shape[0] != a2.shape[1]:
            raise ValueError(f"the decay's low-rank matrices do not fit: {list(a1.shape)} and "
                             f"{list(a2.shape)}")
        self.rank = a1.shape[0]
        self.a1 = Linear(a1.to(device=ctx.device, dtype=ctx.dtype).contiguous())
        self.a2t = f32(a2).t().contiguous()
        self.a2_bias = f32(tensors[self.names["a2_bias"]]).contiguous()

    def _mix(self, x, proj, batch, state, o, out) -> None:
        q, k, v, g = self._split(proj)
        log_decay = torch.empty((x.shape[0], q.shape[1]), dtype=torch.float32, device=x.device)
        ops.lowrank_expand(self.a1(x, out_dtype=torch.float32), 0, self.a2t, log_decay,
                           bias=self.a2_bias, log_decay="sigmoid", rate=1.0 / self.tau)
        ops.channel_scan(q, k, v, log_decay, state, batch.row_start, batch.row_slot, o,
                         batch.n_rows, self.n_heads, self.key_dim, self.value_dim,
                         longest=batch.max_new if batch.n_multi else 1, shortest=batch.min_new,
                         scale=self.key_dim ** -0.5)
        ops.head_norm_gate(o, g, self.gain, self.eps, out, self.n_heads)


@register_mixer("lightning_attention")
class LightningAttention(_LinearAttention):
    def __init__(self, hidden_size: int, n_heads: int, key_dim: int, value_dim: int,
                 decay: Sequence[float], eps: float, names: Mapping[str, str] | None = None) -> None:
        super().__init__(hidden_size, n_heads, key_dim, value_dim, eps, names)
        if len(decay) != n_heads or not all(0.0 <= a <= 1.0 for a in decay):
            raise ValueError(f"decay must give one number from 0 to 1 per head, got {decay!r}")
        self.decay = [float(a) for a in decay]
        self.log_decay = None

    def kernel_jobs(self, dtype: torch.dtype):
        return [ops.core_job("sllm_recurrent_ops"), ops.core_job("sllm_gated_scan")]

    def param_specs(self) -> dict[str, ParamSpec]:
        return {**super().param_specs(),
                self.names["norm"]: ParamSpec((self.n_heads * self.value_dim,), "gain")}

    def load(self, tensors: Mapping[str, torch.Tensor], ctx: BuildContext) -> None:
        super().load(tensors, ctx)
        # (a decay of 0 as one that leaves nothing in 32-bit: sums of its logarithm stay finite)
        self.log_decay = torch.tensor([max(math.log(a), -150.0) if a > 0 else -150.0
                                       for a in self.decay], dtype=torch.float64
                                      ).to(device=ctx.device, dtype=torch.float32)

    def _mix(self, x, proj, batch, state, o, out) -> None:
        q, k, v, g = self._split(proj)
        longest = batch.max_new if batch.n_multi else 1
        # the silu of q, k and v: inside the scan in steps of short rows, else ahead of it
        inside = longest < ops.GATED_SCAN_MIN_CHUNKED
        if not inside:
            ops.silu_columns(proj[:, :self.cols[3]])
        ops.gated_scan(q, k, v, self.log_decay, None, state, batch.row_start, batch.row_slot, o,
                       batch.n_rows, self.n_heads, self.key_dim, self.value_dim, longest=longest,
                       shortest=batch.min_new, silu=inside)
        ops.gate_part_norm(o, g, self.gain, self.eps, 1, out, gate_activation="sigmoid",
                           gate_after=True)
