"""The selective state-space mixer in the Mamba-1 form."""

from __future__ import annotations

import math
from typing import List, Optional

import torch

from .base import Mixer, StateSpec, WeightSpec, register_mixer
from .params import SelectiveScanParams


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class SelectiveScan(Mixer):
    """``wo(y * silu(z))`` with ``y`` the output of a linear recurrence whose every channel keeps ``state``
    numbers with decays of their own.

    ``w_in x`` is ``[x | z]`` (``inner`` columns each).  x passes a causal convolution per channel (``conv``
    taps, the last one on the current token, a bias) and SiLU; ``w_x x`` is then ``[dt | B | C]`` (``dt_rank``,
    ``state``, ``state`` columns).  Per channel c and state number n, in float32:

        d = softplus(w_dt dt + dt_bias);  S[c, n] <- exp(-d_c exp(A_log[c, n])) S[c, n] + d_c x_c B_n
        y_c = sum_n S[c, n] C_n + D_c x_c

    The request's state is fixed-size: S ([inner][state]) and the convolution's last ``conv - 1`` inputs, one
    float32 row per slot that the cache manager zeroes on admission.  The recurrence runs token by token in
    float32, so prompt portions, single tokens and mixed batches take the same kernels and give the same
    numbers however a prompt is cut.
    """

    params: SelectiveScanParams
    graph_safe = True

    def __init__(self, spec) -> None:
        super().__init__(spec)
        p = self.params
        self.scan_floats = p.inner * p.state
        self.conv_floats = (p.conv - 1) * p.inner
        #: where B begins in the rows of the product that gives dt, B and C
        self.b_offset = _pad8(p.dt_rank)

    def weight_specs(self) -> List[WeightSpec]:
        p, n = self.params, self.names
        return [
            WeightSpec(n["w_in"], (2 * p.inner, p.dim)),
            WeightSpec(n["conv"], (p.inner, p.conv), ("normal", 0.3)),
            WeightSpec(n["conv_bias"], (p.inner,), ("normal", 0.1)),
            WeightSpec(n["w_x"], (p.dt_rank + 2 * p.state, p.inner)),
            WeightSpec(n["w_dt"], (p.inner, p.dt_rank)),
            WeightSpec(n["dt_bias"], (p.inner,), ("uniform", -4.0, 0.0)),
            WeightSpec(n["a_log"], (p.inner, p.state), ("uniform", -1.0, 1.5)),
            WeightSpec(n["d"], (p.inner,), ("ones",)),
            WeightSpec(n["wo"], (p.dim, p.inner)),
        ]

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((self.scan_floats + self.conv_floats,))

    def bind(self, tensors, ops) -> None:
        p = self.params
        self.ops = ops
        dt = ops.act_dtype
        self.w_in = tensors["w_in"].to(dt).contiguous()
        # dt's rows are padded to a multiple of 8 and so is the whole, so that views of the product are aligned;
        # the second map of the step sizes has zero columns for the padding
        w_x = tensors["w_x"]
        rows = w_x.new_zeros((_pad8(self.b_offset + 2 * p.state), p.inner))
        rows[: p.dt_rank] = w_x[: p.dt_rank]
        rows[self.b_offset : self.b_offset + 2 * p.state] = w_x[p.dt_rank :]
        self.w_x = rows.to(dt).contiguous()
        w_dt = tensors["w_dt"].new_zeros((p.inner, self.b_offset))
        w_dt[:, : p.dt_rank] = tensors["w_dt"]
        self.w_dt = w_dt.to(dt).contiguous()
        self.wo = tensors["wo"].to(dt).contiguous()
        # what enters float32 arithmetic is float32 whatever it was stored in
        self.conv_w = tensors["conv"].float().contiguous()
        self.conv_b = tensors["conv_bias"].float().contiguous()
        self.dt_bias = tensors["dt_bias"].float().contiguous()
        self.a_log2 = (-torch.exp(tensors["a_log"].float()) * math.log2(math.e)).contiguous()
        self.d = tensors["d"].float().contiguous()

    def forward(self, x, ctx, memory):
        p, ops = self.params, self.ops
        state = memory.state
        proj = ops.linear(x, self.w_in)  # [T, x | z]
        u = ops.time_conv(proj, 0, p.inner, self.conv_w, self.conv_b, state, self.scan_floats, p.conv, ctx, act="silu",
                          out_dtype=x.dtype)
        low = ops.linear(u, self.w_x)  # [T, dt | B | C]
        dt = ops.linear(low[:, : self.b_offset], self.w_dt)
        y = ops.selective_scan(u, dt, low, self.b_offset, proj[:, p.inner :], self.dt_bias, self.a_log2, self.d, state, ctx,
                               p.state)
        return ops.linear(y, self.wo)


register_mixer("selective_scan", SelectiveScan)
