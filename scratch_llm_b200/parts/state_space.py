"""A state-space layer (the SSD form of Mamba-2) as a mixer: a recurrent layer whose state per
request is one matrix ``S`` [state, value] per head in 32-bit, plus the last inputs of a short
convolution.

    [z | x | B | C | dt] = W_in h     (H V | H V | G N | G N | H)
    x, B and C together pass a causal convolution over time per channel (``conv_taps`` taps and
    a bias; the last tap is the current token's, zeros before the start) and silu
    dt = softplus(dt + dt_bias)
    S <- exp(-exp(A_log_h) dt) S + dt B x^T;   y = S^T C + D_h x       (head h reads group
                                                                        h // (H / G))
    out = W_o ( groupnorm(y * silu(z)) * gain )

where groupnorm divides each of ``norm_groups`` equal parts of all heads' channels by its own root
mean square: the gate comes before the norm.

What enters the recurrence besides the projections and the convolution (step sizes, decays, the
state, the read-out) is 32-bit; dt's projection has a 32-bit output.  The state lives in the
cache manager's state slots, so a request may be fed in portions of any size, beside other
requests, and its slot is used again after it ends.
"""

from __future__ import annotations

from typing import Mapping

import torch

from ..kernels import ops
from ..weights.loader import ParamSpec
from .base import BuildContext, CacheView, Mixer, PositionEncoding, StateSpec
from .linear import Linear
from .registry import register_mixer


@register_mixer("state_space")
class StateSpace(Mixer):
    pad_safe = True   # padding tokens belong to no row: the recurrence never sees them

    def __init__(self, hidden_size: int, n_heads: int, n_groups: int, state_dim: int,
                 value_dim: int, conv_taps: int, norm_groups: int, eps: float,
                 names: Mapping[str, str] | None = None) -> None:
        if min(n_heads, n_groups, value_dim, norm_groups) < 1 or n_heads % n_groups:
            raise ValueError(f"{n_heads} heads do not group evenly over {n_groups} groups")
        if (n_heads * value_dim) % norm_groups:
            raise ValueError(f"{n_heads * value_dim} channels do not form {norm_groups} equal "
                             "parts")
        if not 1 <= state_dim <= ops.GATED_SCAN_MAX_KEY_DIM:
            raise ValueError(f"state size {state_dim}: the scan kernel takes 1 to "
                             f"{ops.GATED_SCAN_MAX_KEY_DIM}")
        if not 1 <= conv_taps <= 16:
            raise ValueError(f"the short convolution takes 1 to 16 taps, got {conv_taps}")
        self.hidden_size, self.n_heads, self.n_groups = hidden_size, n_heads, n_groups
        self.state_dim, self.value_dim, self.conv_taps = state_dim, value_dim, conv_taps
        self.norm_groups, self.eps = norm_groups, float(eps)
        self.inner = n_heads * value_dim
        self.names = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias",
                      "A_log": "A_log", "D": "D", "norm": "norm", "o": "o", **(names or {})}
        self.dtype = torch.float32
        self.proj: Linear | None = None      # [x; B; C; z] (zero rows in between, see load)
        self.dt: Linear | None = None        # 32-bit output
        self.o: Linear | None = None
        self.z_col = 0
        self.taps = self.taps_t = self.conv_bias = self.dt_bias = self.a_log = self.skip = None
        self.gain = None

    @property
    def conv_channels(self) -> int:
        return self.inner + 2 * self.n_groups * self.state_dim

    def state_spec(self):
        S = StateSpec((self.n_heads, self.value_dim, self.state_dim), torch.float32)
        if self.conv_taps == 1:
            return S
        return (S, StateSpec((self.conv_taps - 1, self.conv_channels), self.dtype))

    def kernel_jobs(self, dtype: torch.dtype):
        return [ops.core_job("sllm_recurrent_ops"), ops.core_job("sllm_gated_scan")]

    def param_specs(self) -> dict[str, ParamSpec]:
        n, d, H, C = self.names, self.hidden_size, self.n_heads, self.conv_channels
        return {n["in"]: ParamSpec((self.inner + C + H, d)),
                n["conv"]: ParamSpec((C, self.conv_taps), "gain"),
                n["conv_bias"]: ParamSpec((C,), "gain"), n["dt_bias"]: ParamSpec((H,), "gain"),
                n["A_log"]: ParamSpec((H,), "gain"), n["D"]: ParamSpec((H,), "gain"),
                n["norm"]: ParamSpec((self.inner,), "gain"),
                n["o"]: ParamSpec((d, self.inner))}

    def load(self, tensors: Mapping[str, torch.Tensor], ctx: BuildContext) -> None:
        put = lambda t: t.to(device=ctx.device, dtype=ctx.dtype)  # noqa: E731
        f32 = lambda t: t.to(device=ctx.device, dtype=torch.float32).contiguous()  # noqa: E731
        n, C = self.names, self.conv_channels
        self.dtype = ctx.dtype
        z, xbc, dt = put(tensors[n["in"]]).split([self.inner, C, self.n_heads], 0)
        # the convolved channels first, the gate's columns from a 16-byte boundary on
        self.z_col = -(-C // 8) * 8
        self.proj = Linear(torch.cat([xbc, xbc.new_zeros((self.z_col - C, xbc.shape[1])), z,
                                      z.new_zeros((-(self.z_col + self.inner) % 8, z.shape[1]))],
                                     0).contiguous())
        self.dt = Linear(dt.contiguous())
        self.o = Linear(put(tensors[n["o"]]).contiguous())
        self.taps = f32(tensors[n["conv"]])
        self.taps_t = self.taps.t().contiguous()
        self.conv_bias, self.dt_bias = f32(tensors[n["conv_bias"]]), f32(tensors[n["dt_bias"]])
        self.a_log, self.skip = f32(tensors[n["A_log"]]), f32(tensors[n["D"]])
        self.gain = f32(tensors[n["norm"]])

    def forward(self, x, batch, cache: CacheView, write: bool, position: PositionEncoding):
        if not write:
            raise NotImplementedError("a run that only reads another run's recurrent state")
        H, G, N, V, C = (self.n_heads, self.n_groups, self.state_dim, self.value_dim,
                         self.conv_channels)
        S, carried = cache.state if isinstance(cache.state, tuple) else (cache.state, None)
        n = x.shape[0]
        proj = self.proj(x)                                        # [N, C | z]
        dt = self.dt(x, out_dtype=torch.float32)                   # [N, H]
        act = torch.empty((n, C), dtype=proj.dtype, device=proj.device)
        ops.conv_silu(proj, self.taps, carried, batch.token_row, batch.row_start, batch.row_slot,
                      act, self.taps_t, bias=self.conv_bias)
        ops.conv_state_update(proj, self.conv_taps, carried, batch.row_start, batch.row_slot,
                              batch.n_rows)
        gates = torch.empty((2, n, H), dtype=torch.float32, device=proj.device)
        ops.ssd_gates(dt, self.dt_bias, self.a_log, gates[0], gates[1])
        # (padding tokens belong to no row: their read-out stays zero)
        y = (torch.zeros if batch.padded else torch.empty)((n, self.inner), dtype=torch.float32,
                                                           device=proj.device)
        ops.gated_scan(act[:, self.inner + G * N:], act[:, self.inner:self.inner + G * N],
                       act[:, :self.inner], gates[0], gates[1], S, batch.row_start,
                       batch.row_slot, y, batch.n_rows, G, N, V,
                       longest=batch.max_new if batch.n_multi else 1,
                       shortest=batch.min_new, skip=self.skip)
        out = torch.empty((n, self.inner), dtype=proj.dtype, device=proj.device)
        ops.gate_part_norm(y, proj[:, self.z_col:self.z_col + self.inner], self.gain, self.eps,
                           self.norm_groups, out)
        return self.o(out)
