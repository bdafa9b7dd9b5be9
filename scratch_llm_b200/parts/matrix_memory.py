"""A matrix memory with exponential gates (the mLSTM of xLSTM) as a mixer: a recurrent layer whose
state per request is one matrix ``S`` [key, value] and one normaliser ``n`` [key] per head, kept
in range by a running maximum ``m``, all in 32-bit:

    q = W_q h * key_dim^(-1/2),  k = W_k h   (H x key_dim),   v = W_v h   (H x value_dim)
    i = cap tanh((W_i h + b_i) / cap),   f = log sigmoid(cap tanh((W_f h + b_f) / cap))
    m' = max(f + m, i)                                          (m starts at 0)
    S <- exp(f + m - m') S + exp(i - m') k v^T,   n likewise with k alone
    o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)
    out = W_o ( rmsnorm_per_head(o) * gain * sigmoid(W_g h) )   (gain: one entry per channel of
                                                                 all heads)

The normaliser is one more column of S (a value that is always 1), so that one scan carries both.
What enters the recurrence besides the projections (gates, their logarithms and exponentials, the
state, the read-out) is 32-bit; the gates' projections have a 32-bit output.  The state lives in
the cache manager's state slots, so a request may be fed in portions of any size, beside other
requests, and its slot is used again after it ends.
"""

from __future__ import annotations

import math
from typing import Mapping

import torch

from ..kernels import ops
from ..weights.loader import ParamSpec
from .base import BuildContext, CacheView, Mixer, PositionEncoding, StateSpec
from .linear import Linear
from .registry import register_mixer


@register_mixer("matrix_memory")
class MatrixMemory(Mixer):
    pad_safe = True   # padding tokens belong to no row: the recurrence never sees them

    def __init__(self, hidden_size: int, n_heads: int, key_dim: int, value_dim: int,
                 gate_cap: float, eps: float, names: Mapping[str, str] | None = None) -> None:
        if min(n_heads, value_dim) < 1:
            raise ValueError("matrix memory: sizes must be positive")
        if not 1 <= key_dim <= ops.GATED_SCAN_MAX_KEY_DIM:
            raise ValueError(f"key size {key_dim}: the scan kernel takes 1 to "
                             f"{ops.GATED_SCAN_MAX_KEY_DIM}")
        if not (gate_cap > 0 and math.isfinite(gate_cap)):
            raise ValueError(f"gate_cap must be positive, got {gate_cap!r}")
        self.hidden_size, self.n_heads = hidden_size, n_heads
        self.key_dim, self.value_dim = key_dim, value_dim
        self.gate_cap, self.eps = float(gate_cap), float(eps)
        self.names = {"q": "q", "k": "k", "v": "v", "g": "g", "o": "o", "norm": "norm", "i": "i",
                      "i_bias": "i.b", "f": "f", "f_bias": "f.b", **(names or {})}
        self.proj: Linear | None = None      # [q; k; v; g] (zero rows in between, see load)
        self.gates: Linear | None = None     # [i; f], 32-bit output
        self.o: Linear | None = None
        self.cols: list[int] = []            # where q, k, v and g start
        self.i_bias = self.f_bias = self.gain = None

    def state_spec(self):
        H = self.n_heads
        return (StateSpec((H, self.value_dim + 1, self.key_dim), torch.float32),
                StateSpec((H,), torch.float32))

    def kernel_jobs(self, dtype: torch.dtype):
        return [ops.core_job("sllm_recurrent_ops"), ops.core_job("sllm_gated_scan")]

    def param_specs(self) -> dict[str, ParamSpec]:
        n, d, H = self.names, self.hidden_size, self.n_heads
        hk, hv = H * self.key_dim, H * self.value_dim
        return {n["q"]: ParamSpec((hk, d)), n["k"]: ParamSpec((hk, d)), n["v"]: ParamSpec((hv, d)),
                n["g"]: ParamSpec((hv, d)), n["o"]: ParamSpec((d, hv)),
                n["norm"]: ParamSpec((hv,), "gain"), n["i"]: ParamSpec((H, d)),
                n["i_bias"]: ParamSpec((H,), "gain"), n["f"]: ParamSpec((H, d)),
                n["f_bias"]: ParamSpec((H,), "gain")}

    def load(self, tensors: Mapping[str, torch.Tensor], ctx: BuildContext) -> None:
        put = lambda t: t.to(device=ctx.device, dtype=ctx.dtype)  # noqa: E731
        f32 = lambda t: t.to(device=ctx.device, dtype=torch.float32).contiguous()  # noqa: E731
        n = self.names
        blocks, at = [], 0
        self.cols = []
        for name in "qkvg":              # each starts on a 16-byte boundary
            w = put(tensors[n[name]])
            self.cols.append(at)
            blocks += [w, w.new_zeros((-w.shape[0] % 8, w.shape[1]))]
            at += -(-w.shape[0] // 8) * 8
        self.proj = Linear(torch.cat(blocks, 0).contiguous())
        self.gates = Linear(torch.cat([put(tensors[n["i"]]), put(tensors[n["f"]])], 0).contiguous())
        self.o = Linear(put(tensors[n["o"]]).contiguous())
        self.i_bias, self.f_bias = f32(tensors[n["i_bias"]]), f32(tensors[n["f_bias"]])
        self.gain = f32(tensors[n["norm"]])

    def forward(self, x, batch, cache: CacheView, write: bool, position: PositionEncoding):
        if not write:
            raise NotImplementedError("a run that only reads another run's recurrent state")
        H, D, V = self.n_heads, self.key_dim, self.value_dim
        S, running = cache.state
        n = x.shape[0]
        proj = self.proj(x)
        pre = self.gates(x, out_dtype=torch.float32)               # [N, 2 H]
        q, k, v, g = (proj[:, c:c + w] for c, w in zip(self.cols, (H * D, H * D, H * V, H * V)))
        one_each = batch.n_multi == 0
        # (padding tokens belong to no row: their gates and read-outs stay zero)
        make = torch.zeros if batch.padded else torch.empty
        gates = make((4, n, H), dtype=torch.float32, device=proj.device)
        log_decay, weight, floor, den = gates
        ops.memory_gates(pre, self.i_bias, self.f_bias, self.gate_cap, running, batch.row_start,
                         batch.row_slot, batch.n_rows, log_decay, weight, floor,
                         one_each=one_each)
        o = make((n, H * V), dtype=torch.float32, device=proj.device)
        ops.gated_scan(q, k, v, log_decay, weight, S, batch.row_start, batch.row_slot, o,
                       batch.n_rows, H, D, V, longest=1 if one_each else batch.max_new,
                       shortest=batch.min_new,
                       ones_out=den, scale=D ** -0.5)
        out = torch.empty((n, H * V), dtype=proj.dtype, device=proj.device)
        ops.head_norm_gate(o, g, self.gain, self.eps, out, H, gate_activation="sigmoid",
                           divisor=(den, floor))
        return self.o(out)
