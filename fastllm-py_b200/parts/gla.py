"""Gated linear attention mixer: linear attention whose state decays per key channel by a number
made from the token; no softmax and no denominator.

For a head with state S [dim x vdim] (float, one per request, zero at the start):

    alpha = sigmoid(W_a2 (W_a1 h) + b_a2)^(1 / tau)            one number per head and key channel
    S <- diag(alpha) S + k v^T;   o = S^T (q * q_scale)        q_scale dim^-1/2 unless given

q, k (`heads` x `dim`) and v (`heads` x `vdim`) are projections of the input.  Each head's o is divided by
its root mean square over vdim and multiplied by a weight [vdim] that the heads share; the heads are
concatenated, multiplied by silu(W_g h) and projected by W_o.

One stacked matrix serves q | k | v | gate | the decay's low-rank input; the small second matrix of the
decay is applied in float by the preparing kernel.  The request's state row holds S for every head; it
is float and carried from step to step by the cache manager's state slots.  Everything after the
projection is float.
"""
from __future__ import annotations

import torch

from ..cache.needs import FixedState
from ..native import ops
from .base import ProjectedMixer
from .registry import register_part


@register_part("mixer", "gated_linear_attention")
class GatedLinearAttention(ProjectedMixer):
    """params: hidden_size, heads, dim, vdim, tau, norm_eps, q_scale (None: dim^-1/2).  tensors: q, k [heads * dim, hidden],
    v, g [heads * vdim, hidden], a1 [rank, hidden], a2 [heads * dim, rank], a2_bias [heads * dim], norm [vdim],
    o [hidden, heads * vdim]; `rank` is a1's row count, a parameter too."""
    category = "mixer"
    native_libraries = ("gla",)
    in_slots = ("q", "k", "v", "g", "a1")
    workspace_name = "gla"

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.heads, self.dim, self.vdim = int(p["heads"]), int(p["dim"]), int(p["vdim"])
        self.rank = int(p["rank"])
        self.tau = float(p["tau"])
        self.norm_eps = float(p["norm_eps"])
        self.q_scale = float(p["q_scale"]) if p.get("q_scale") is not None else self.dim ** -0.5
        if self.dim > 256:
            raise ValueError(f"gated_linear_attention: dim {self.dim} is beyond the scan kernel's limit of 256")
        self.hd, self.hv = self.heads * self.dim, self.heads * self.vdim
        self.in_cols, self.out_cols = 2 * self.hd + 2 * self.hv + self.rank, self.hv     # q | k | v | gate | low

    def cache_need(self):
        return FixedState((self.heads * self.vdim * self.dim,), "float32")

    def in_rows(self):
        return {"q": self.hd, "k": self.hd, "v": self.hv, "g": self.hv, "a1": self.rank}

    def core_shapes(self):
        return {"a2": (self.hd, self.rank), "a2_bias": (self.hd,), "norm": (self.vdim,)}

    def load_core(self, tensors):
        self.a2 = tensors["a2"].float().t().contiguous()               # [rank, heads * dim]: the kernel reads along heads * dim
        self.a2_bias = tensors["a2_bias"].float().contiguous()
        self.norm_w = tensors["norm"].contiguous()
        if self.result_scale != 1.0:
            self.norm_w = (self.norm_w.double() * self.result_scale).float()

    def core(self, proj, y, step, cache):
        n = proj.shape[0]
        ws = step.workspace
        work = ws.rows("gla_work", n, 3 * self.hd + self.hv, torch.float32)
        ops.gla_prep(proj, self.a2, self.a2_bias, work, self.heads, self.dim, self.vdim, self.rank, self.q_scale, self.tau)
        o = ws.rows("gla_o", n, self.hv, torch.float32)
        ops.gla_scan(work, o, cache.tensor, step, self.heads, self.dim, self.vdim)
        ops.gla_gated_norm(o, proj[:, 2 * self.hd + self.hv:2 * self.hd + 2 * self.hv], self.norm_w, y, self.heads,
                           self.vdim, self.norm_eps)
