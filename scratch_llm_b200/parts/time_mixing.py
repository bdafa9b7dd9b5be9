"""Time mixing with a bonus (the recurrence of RWKV) as a mixer: a recurrent layer whose state per
request is one matrix ``S`` [key, value] per head and the previous token's input, both in 32-bit.

    with h' the previous token's h (zeros for a sequence's first token), each of r, k, v, g and w reads
    its own mix  m_s = h + (h' - h) * mu_s
    r, k, v = W_r m_r, W_k m_k, W_v m_v  (H x dim)        gate = silu(W_g m_g)
    w = exp(-exp(W_w2 tanh(W_w1 m_w) + w0))               (the decay, per head and key channel)
    o = (S + diag(u) k v^T)^T r                           (the bonus u weighs the token's own write)
    S <- diag(w) S + k v^T
    out = W_o ( rmsnorm_per_head(o) * gain * gate )       (gain: one entry per channel of all heads)

One kernel forms the five mixes; the four wide projections, each with an input of its own, share a
launch.  The low-rank path from its first product's output on, the decay, the state and the read-out
are 32-bit.  The state lives in the cache manager's state slots, so a request may be fed in portions
of any size, beside other requests, and its slot is used again after it ends.
"""

from __future__ import annotations

from typing import Mapping

import torch

from ..kernels import ops
from ..weights.loader import ParamSpec
from .base import BuildContext, CacheView, Mixer, PositionEncoding, StateSpec
from .linear import GroupedLinear, Linear
from .registry import register_mixer


@register_mixer("time_mixing")
class TimeMixing(Mixer):
    pad_safe = True   # padding tokens belong to no row: the recurrence never sees them

    def __init__(self, hidden_size: int, n_heads: int, head_dim: int, eps: float,
                 decay_rank: int = -1, names: Mapping[str, str] | None = None) -> None:
        """``decay_rank``: the low rank of the decay's pair of matrices (-1: as the tensors say)."""
        if n_heads < 1 or not 1 <= head_dim <= ops.GATED_SCAN_MAX_KEY_DIM:
            raise ValueError(f"time mixing: heads {n_heads} of {head_dim} (the scan kernel takes "
                             f"sizes 1 to {ops.GATED_SCAN_MAX_KEY_DIM})")
        self.hidden_size, self.n_heads, self.dim = hidden_size, n_heads, head_dim
        self.eps, self.rank = float(eps), decay_rank
        self.names = {**{n: n for n in ("r", "k", "v", "g", "o", "w1", "w2", "w0", "u", "norm")},
                      **{f"mu_{n}": f"mu.{n}" for n in "rkvgw"}, **(names or {})}
        self.wide: GroupedLinear | None = None     # r, k, v, g
        self.w1: Linear | None = None              # 32-bit output
        self.o: Linear | None = None
        self.mu = self.w2t = self.w0 = self.u = self.gain = None

    def state_spec(self):
        return (StateSpec((self.n_heads, self.dim, self.dim), torch.float32),
                StateSpec((self.hidden_size,), torch.float32))

    def kernel_jobs(self, dtype: torch.dtype):
        return [ops.core_job("sllm_recurrent_ops"), ops.core_job("sllm_channel_scan")]

    def param_specs(self) -> dict[str, ParamSpec]:
        n, d, hd = self.names, self.hidden_size, self.n_heads * self.dim
        specs = {n[c]: ParamSpec((hd, d)) for c in "rkvg"}
        specs.update({n[f"mu_{c}"]: ParamSpec((d,), "gain") for c in "rkvgw"})
        specs.update({n["w1"]: ParamSpec((self.rank, d)), n["w2"]: ParamSpec((hd, self.rank)),
                      n["w0"]: ParamSpec((hd,), "gain"),
                      n["u"]: ParamSpec((self.n_heads, self.dim), "gain"),
                      n["norm"]: ParamSpec((hd,), "gain"), n["o"]: ParamSpec((d, hd))})
        return specs

    def load(self, tensors: Mapping[str, torch.Tensor], ctx: BuildContext) -> None:
        put = lambda t: t.to(device=ctx.device, dtype=ctx.dtype)  # noqa: E731
        f32 = lambda t: t.to(device=ctx.device, dtype=torch.float32).contiguous()  # noqa: E731
        n = self.names
        w1, w2 = tensors[n["w1"]], tensors[n["w2"]]
        if w1.shape[0] != w2.shape[1]:
            raise ValueError(f"the decay's low-rank matrices do not fit: {list(w1.shape)} and "
                             f"{list(w2.shape)}")
        self.rank = w1.shape[0]
        self.wide = GroupedLinear(torch.stack([put(tensors[n[c]]) for c in "rkvg"]).contiguous())
        self.w1 = Linear(put(w1).contiguous())
        self.o = Linear(put(tensors[n["o"]]).contiguous())
        self.mu = torch.stack([f32(tensors[n[f"mu_{c}"]]) for c in "rkvgw"]).contiguous()
        self.w2t, self.w0 = f32(w2).t().contiguous(), f32(tensors[n["w0"]])
        self.u, self.gain = f32(tensors[n["u"]]), f32(tensors[n["norm"]])

    def forward(self, x, batch, cache: CacheView, write: bool, position: PositionEncoding):
        return self.o(self.heads_out(x, batch, cache, write, position))

    def heads_out(self, x, batch, cache: CacheView, write: bool, position: PositionEncoding,
                  out: torch.Tensor | None = None) -> torch.Tensor:
        """The heads' read-outs, normed and gated [N, H * dim]: what the output matrix multiplies.
        ``out``: where to put them (may be a column slice)."""
        if not write:
            raise NotImplementedError("a run that only reads another run's recurrent state")
        H, D = self.n_heads, self.dim
        S, carried = cache.state
        n, hd = x.shape[0], H * D
        mixes = torch.empty((5, n, self.hidden_size), dtype=x.dtype, device=x.device)
        ops.shift_mix(x, self.mu, carried, batch.token_row, batch.row_start, batch.row_slot, mixes)
        r, k, v, g = self.wide(mixes[:4])
        log_decay = torch.empty((n, hd), dtype=torch.float32, device=x.device)
        ops.lowrank_expand(self.w1(mixes[4], out_dtype=torch.float32), 0, self.w2t, log_decay,
                           bias=self.w0, log_decay="exp", tanh_in=True)
        # (padding tokens belong to no row: their read-out stays zero)
        o = (torch.zeros if batch.padded else torch.empty)((n, hd), dtype=torch.float32,
                                                           device=x.device)
        ops.channel_scan(r, k, v, log_decay, S, batch.row_start, batch.row_slot, o, batch.n_rows,
                         H, D, D, longest=batch.max_new if batch.n_multi else 1,
                         shortest=batch.min_new, bonus=self.u)
        if out is None:
            out = torch.empty((n, hd), dtype=x.dtype, device=x.device)
        ops.head_norm_gate(o, g, self.gain, self.eps, out, H)
        return out

    # -- for a block or mixer that multiplies several branches' activations by one joined matrix

    def out_segments(self):
        """[(the output matrix [hidden, H * dim], its weight in the layer's sum)]."""
        return [(self.o.weight, 1.0)]

    def scale_activations(self, factor: float) -> None:
        """Multiply what activations_into writes by ``factor`` from now on (in 32-bit, ahead of its
        rounding: the gain takes it)."""
        self.gain = self.gain * float(factor)

    def release_out(self) -> None:
        self.o = None

    def activations_into(self, x, batch, cache: CacheView, write: bool, position, outs) -> None:
        self.heads_out(x, batch, cache, write, position, out=outs[0])
