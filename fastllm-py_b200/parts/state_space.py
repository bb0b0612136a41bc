"""State-space mixer: a matrix state per head that decays by one number per token, written and read through
vectors that groups of heads share (a selective state space in its "duality" form).

One stacked product gives [z: inner | x: inner | B: groups x state | C: groups x state | dt: heads] with
inner = heads x vdim; head h uses group h // (heads / groups):

    x, B, C <- silu(conv(x, B, C) + bias)         one causal convolution per channel, `taps` taps
    dt <- softplus(dt + dt_bias)
    S <- exp(-exp(A_log) dt) S + dt B x^T;   y = S^T C + D x          (S: state x vdim per head)
    out = W_o (norm(y * silu(z)) * weight)        norm: an RMS norm in `norm_parts` equal parts of inner

The request's state row holds S for every head and behind it the convolution's last taps - 1 inputs; it is float
and carried from step to step by the cache manager's state slots.  Everything after the product is float.  Steps of
single tokens run the mixer up to the norm in one kernel; prompt portions and mixed steps (and every step of the
32-bit path, so that cuts and batches agree bit for bit) prepare all tokens first and then walk each request's.
"""
from __future__ import annotations

import torch

from ..cache.needs import FixedState
from ..native import ops
from .base import ProjectedMixer
from .registry import register_part


@register_part("mixer", "state_space")
class StateSpace(ProjectedMixer):
    """params: hidden_size, heads, vdim, state, groups, taps, norm_parts, norm_eps.  tensors: in [2 heads * vdim +
    2 groups * state + heads, hidden], conv [heads * vdim + 2 groups * state, taps], conv_bias, dt_bias, A_log, D [heads],
    norm [heads * vdim], o [hidden, heads * vdim]."""
    category = "mixer"
    native_libraries = ("ssd",)
    in_slots = ("in",)
    workspace_name = "state_space"

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.heads, self.vdim, self.state = int(p["heads"]), int(p["vdim"]), int(p["state"])
        self.groups, self.taps, self.parts = int(p["groups"]), int(p["taps"]), int(p["norm_parts"])
        self.norm_eps = float(p["norm_eps"])
        self.inner = self.heads * self.vdim
        if self.heads % self.groups:
            raise ValueError(f"state_space: {self.heads} heads are not a multiple of {self.groups} groups")
        if self.inner % self.parts:
            raise ValueError(f"state_space: {self.parts} norm parts do not divide the inner width {self.inner}")
        if self.state > 256:
            raise ValueError(f"state_space: state {self.state} is beyond the kernels' limit of 256")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"state_space: {self.taps} taps are beyond the kernels' 16")
        self.channels = self.inner + 2 * self.groups * self.state          # what passes the convolution: x | B | C
        self.in_cols, self.out_cols = self.inner + self.channels + self.heads, self.inner
        self.state_floats = self.inner * self.state

    def cache_need(self):
        floats = self.state_floats + (self.taps - 1) * self.channels
        return FixedState((-(-floats // 4) * 4,), "float32")               # (rows that start on 16 bytes)

    def in_rows(self):
        return {"in": self.in_cols}

    def core_shapes(self):
        h = (self.heads,)
        return {"conv": (self.channels, self.taps), "conv_bias": (self.channels,), "dt_bias": h, "A_log": h, "D": h,
                "norm": (self.inner,)}

    def load_core(self, tensors):
        self.conv_w = tensors["conv"].float().t().contiguous()             # [taps, channels]: read along the channels
        self.conv_b = tensors["conv_bias"].float().contiguous()
        self.dt_bias = tensors["dt_bias"].float().contiguous()
        self.neg_a = (-torch.exp(tensors["A_log"].double())).contiguous()
        self.skip = tensors["D"].float().contiguous()
        self.norm_w = (tensors["norm"].double() * self.result_scale).float().contiguous()

    def core(self, proj, y, step, cache):
        n = proj.shape[0]
        ws = step.workspace
        rows = cache.tensor
        tail = rows[:, self.state_floats:] if self.taps > 1 else None
        out = ws.rows("state_space_out", n, self.inner, torch.float32)
        sizes = (self.heads, self.vdim, self.state, self.groups)
        if self.ctx.dtype == torch.bfloat16 and n == step.n_requests:
            ops.ssd_step(proj, self.conv_w, self.conv_b, self.dt_bias, self.neg_a, self.skip, out, rows, self.state_floats,
                         step, *sizes)
        else:
            work = ws.rows("state_space_work", n, self.channels + 2 * self.heads, torch.float32)
            ops.ssd_prep(proj, self.conv_w, self.conv_b, self.dt_bias, self.neg_a, tail, step, work, *sizes)
            ops.ssd_scan(work, self.skip, out, rows, step, *sizes)
        ops.ssd_norm(out, proj, self.norm_w, y, self.parts, self.norm_eps, tail, self.taps, self.channels, step)
