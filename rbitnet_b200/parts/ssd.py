"""``StateSpace``: a mixer that keeps a state S [state_dim, value_dim] per head and forgets it at one rate per head and
token (the recurrence of Mamba-2, "Transformers are SSMs", Dao and Gu).

From the input rows h, one stacked projection W_in h = [z | x | B | C | dt]: z and x have ``n_heads`` heads of
``value_dim`` values, B and C ``n_groups`` vectors of ``state_dim`` values (head i reads group i // (n_heads / n_groups)),
dt one number per head.  x, B and C together go through a short causal convolution per channel ("conv": [channels, taps],
the last tap is the current token's, zeros before the start of the sequence; bias "conv.b") and SiLU.  Then, per head,

    d = softplus(dt + dt_bias)
    S <- exp(-exp(A_log) d) S + d B x^T;   y = S^T C + D x                            (the read-out sees the write)
    result = W_o (rms_in_groups(y * silu(z)) * w)        (``norm_groups`` equal parts of the joined heads, each divided by its
                                                          own root mean square; w spans them all)

State per sequence: S (float32, [heads, state_dim, value_dim]) and the convolution's last inputs as a ring of ``taps``
rows by position.  Step sizes, decays, the state and its sums, the gate and the norm are float32 in every mode; the
projection leaves float32 rows.
"""
from __future__ import annotations

import torch

from .base import Mixer, StateNeed
from .registry import register_part


class StateSpace(Mixer):
    def __init__(self, width: int, n_heads: int, value_dim: int, state_dim: int, n_groups: int, taps: int,
                 norm_groups: int, norm_eps: float):
        self.width, self.n_heads, self.value_dim = int(width), int(n_heads), int(value_dim)
        self.state_dim, self.n_groups, self.taps = int(state_dim), int(n_groups), int(taps)
        self.norm_groups, self.norm_eps = int(norm_groups), float(norm_eps)
        if min(self.n_heads, self.value_dim, self.state_dim, self.n_groups, self.taps, self.norm_groups) < 1:
            raise ValueError("state space: heads, sizes, groups and taps are at least 1")
        if self.n_heads % self.n_groups:
            raise ValueError(f"state space: {n_heads} heads are not a multiple of {n_groups} groups")
        if (self.n_heads * self.value_dim) % self.norm_groups:
            raise ValueError(f"state space: {n_heads} heads of {value_dim} values are not {norm_groups} equal parts")
        self.w_in = self.w_o = self.conv_w = self.conv_b = None
        self.a_log = self.dt_bias = self.d_skip = self.norm_w = None

    @property
    def channels(self) -> int:
        """Channels that are convolved: x, B and C."""
        return self.n_heads * self.value_dim + 2 * self.n_groups * self.state_dim

    def weight_shapes(self):
        H, E, K, C = self.n_heads, self.width, self.taps, self.channels
        inner = H * self.value_dim
        return {"in": ((inner + C + H, E), "matrix"), "conv": ((C, K), "taps"), "conv.b": ((C,), "matrix"),
                "dt_bias": ((H,), "matrix"), "A_log": ((H,), "matrix"), "D": ((H,), "norm"), "norm": ((inner,), "norm"),
                "o": ((E, inner), "matrix")}

    def state_need(self):
        need = {"S": StateNeed((self.n_heads, self.state_dim, self.value_dim))}
        if self.taps > 1:
            need["tail"] = StateNeed((self.taps, self.channels))
        return need

    def offsets(self):
        """Columns of the stacked product's rows."""
        inner = self.n_heads * self.value_dim
        return {"z": 0, "x": inner, "dt": inner + self.channels}

    def bind(self, weights, ops):
        w = weights["in"]
        pad = -w.shape[0] % 8
        if pad:                                    # rows whose length allows 16-byte accesses
            w = torch.cat([w, torch.zeros((pad, w.shape[1]), dtype=w.dtype, device=w.device)], dim=0)
        self.w_in = ops.prepare_linear([w])
        self.w_o = ops.prepare_linear([weights["o"]])
        f32 = dict(device=ops.device, dtype=torch.float32)
        self.conv_w, self.conv_b = (weights[k].to(**f32).contiguous() for k in ("conv", "conv.b"))
        self.a_log, self.dt_bias, self.d_skip, self.norm_w = (
            weights[k].to(**f32).contiguous() for k in ("A_log", "dt_bias", "D", "norm"))

    def forward(self, ctx, h, entry, accumulate_into=None):
        ops = ctx.ops
        proj = ops.linear(h, self.w_in, out_dtype=torch.float32)               # [T, z | x | B | C | dt | padding]
        v = ops.state_space(proj, self, ctx.state_view(entry), ctx.meta)       # [T, H value_dim], float32: y silu(z)
        out = ops.rmsnorm_grouped(v, self.norm_w, self.norm_groups, self.norm_eps)
        if accumulate_into is None:
            return ops.linear(out, self.w_o, out_dtype=torch.float32)
        return ops.linear(out, self.w_o, accumulate_into=accumulate_into)


register_part("mixer", "state_space", StateSpace)
