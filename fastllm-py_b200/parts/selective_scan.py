"""Selective scan mixer: a recurrence per channel and state element whose decay is made from the token for every one of
them (the first form of a selective state space).

One product gives [u: inner | z: inner]:

    x <- silu(conv(u) + bias)                      one causal convolution per channel, `taps` taps
    [dt: rank | B: state | C: state] = W_x x;      dt <- softplus(W_dt dt + bias), one number a channel
    S[c, n] <- exp(-exp(A_log[c, n]) dt_c) S[c, n] + dt_c x_c B_n;      y_c = sum_n S[c, n] C_n + D_c x_c
    out = W_o (y * silu(z))

The request's state row holds S [inner, state] and behind it the convolution's last taps - 1 inputs; it is float and
carried from step to step by the cache manager's state slots.  x is of the activation type; W_x's result, dt, decays, the
state and the read-out are float.  Steps of single tokens take two kernels beside the small product; prompt portions and
mixed steps (and every step of the 32-bit path, so that cuts and batches agree bit for bit) prepare all tokens first and
then walk each request's.
"""
from __future__ import annotations

import math

import torch

from ..cache.needs import FixedState
from ..native import ops
from .base import ProjectedMixer
from .linear import Linear
from .registry import register_part


@register_part("mixer", "selective_scan")
class SelectiveScan(ProjectedMixer):
    """params: hidden_size, inner, state, rank, taps.  tensors: in [2 inner, hidden], conv [inner, taps], conv_bias [inner],
    x [rank + 2 state, inner], dt [inner, rank], dt_bias [inner], A_log [inner, state], D [inner], o [hidden, inner]."""
    category = "mixer"
    native_libraries = ("selective_scan",)
    in_slots = ("in",)
    workspace_name = "selective"

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        p = spec.params
        self.hidden, self.inner = int(p["hidden_size"]), int(p["inner"])
        self.state, self.rank, self.taps = int(p["state"]), int(p["rank"]), int(p["taps"])
        if self.state > 256:
            raise ValueError(f"selective_scan: state {self.state} is beyond the kernels' limit of 256")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"selective_scan: {self.taps} taps are beyond the kernels' 16")
        if self.rank > 8192:
            raise ValueError(f"selective_scan: rank {self.rank} is beyond the kernels' limit of 8192")
        self.low_cols = self.rank + 2 * self.state
        self.in_cols, self.out_cols = 2 * self.inner, self.inner
        self.state_floats = -(-self.inner * self.state // 4) * 4              # (the kept inputs start on 16 bytes)
        self.low = self.dt = None

    def cache_need(self):
        floats = self.state_floats + (self.taps - 1) * self.inner
        return FixedState((-(-floats // 4) * 4,), "float32")

    def in_rows(self):
        return {"in": 2 * self.inner}

    def core_shapes(self):
        n = (self.inner,)
        return {"conv": (self.inner, self.taps), "conv_bias": n, "x": (self.low_cols, self.inner), "dt": (self.inner, self.rank),
                "dt_bias": n, "A_log": (self.inner, self.state), "D": n}

    def load_core(self, tensors):
        self.low = Linear([tensors["x"]])
        self.conv_w = tensors["conv"].float().t().contiguous()                # [taps, inner]: read along the channels
        self.conv_b = tensors["conv_bias"].float().contiguous()
        w = tensors["dt"]
        pitch = -(-self.rank // 8) * 8
        self.dt_w = torch.zeros((self.inner, pitch), dtype=w.dtype, device=w.device)      # rows that start on 16 bytes
        self.dt_w[:, :self.rank] = w
        # prompt portions: W_dt twice over, against the two bfloat16 parts of a float row, where the product is bfloat16
        self.split = self.ctx.dtype == torch.bfloat16 and w.dtype == torch.bfloat16
        self.dt = Linear([torch.cat([w, w], dim=1) if self.split else w])
        self.dt_bias = tensors["dt_bias"].float().contiguous()
        a = -torch.exp(tensors["A_log"].double())
        self.a = (a * math.log2(math.e) if self.ctx.dtype == torch.bfloat16 else a).float().contiguous()
        self.skip = tensors["D"].float().contiguous()

    def reserve(self, limits):
        super().reserve(limits)
        self.low.reserve(self.ctx.dtype, limits.max_tokens)
        if self.split:
            self.dt.reserve(self.ctx.dtype, limits.max_tokens)

    def core(self, proj, y, step, cache):
        n = proj.shape[0]
        ws = step.workspace
        rows = cache.tensor
        tail = rows[:, self.state_floats:] if self.taps > 1 else None
        u, z = proj[:, :self.inner], proj[:, self.inner:]
        single = self.ctx.dtype == torch.bfloat16 and n == step.n_requests
        x = ws.rows("selective_x", n, self.inner, self.ctx.dtype)
        ops.selective_conv(u, self.conv_w, self.conv_b, tail, step, x, single)
        low = ws.rows("selective_low", n, self.low_cols, torch.float32)
        left = self.low.forward(x, low, defer=single)
        if single:
            ops.selective_step(x, z, low if left is None else left, self.rank, self.dt_w, self.dt_bias, self.a, self.skip,
                               self.result_scale, y, rows, step)
            return
        dt = ws.rows("selective_dt", n, self.inner, torch.float32)
        if self.split:
            parts = ws.rows("selective_parts", n, 2 * self.rank, torch.bfloat16)
            ops.selective_split(low, self.rank, parts)
            self.dt.forward(parts, dt)
        else:
            self.dt.forward(low[:, :self.rank], dt)
        ops.selective_scan(x, z, u, dt, self.dt_bias, low, self.rank, self.a, self.skip, self.result_scale, y, rows,
                           self.state_floats, self.taps, step)
