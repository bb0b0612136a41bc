"""Two mixers side by side: both read the same input, and the layer's result is the weighted sum of
their results, each first normed over the model width.

    out = weight * (rms(left(h)) * w_left + rms(right(h)) * w_right)       (weight 1/2: their average)

Each of the two is a mixer part of its own with whatever cache or state it needs; this part asks the
cache manager for both (`cache_needs`) and hands each its view.  Either may leave its last product as
split-K partial sums, which the one kernel that norms both rows and mixes them adds up as it reads.
The scratch for partial sums is one buffer and a second one beside it: a left mixer that says
`honours_partial_side` is told (`partial_side = True`) to leave its sums in the second, where the right
mixer's products do not overwrite them; one that does not gets its sums added up before the right runs.

"side_by_side_sum" is the plain weighted sum of two mixers, which then share their two matrix products.
"""
from __future__ import annotations

import torch

from ..native import ops
from .base import Part, ProjectedMixer
from .linear import Linear
from .plan import PartSpec
from .registry import build_part, register_part


def side_needs(side: str, part) -> dict:
    """name -> need of one side's mixer: `side` for its one need, `side.<name>` for each of several."""
    need = part.cache_need()
    needs = {} if need is None else {side: need}
    for name, sub in (part.cache_needs() if hasattr(part, "cache_needs") else {}).items():
        needs[f"{side}.{name}"] = sub
    return needs


def side_view(side: str, part, views):
    """What one side's mixer is handed: its one view, or its views by name."""
    if views is None:
        return None
    names = part.cache_needs() if hasattr(part, "cache_needs") else ()
    return {name: views.get(f"{side}.{name}") for name in names} if names else views.get(side)


class Sides(Part):
    """What two mixers on one input have in common: they are children, their needs and what they decide per step are
    asked for through this part."""
    category = "mixer"
    SIDES = ("left", "right")
    left = right = None

    def children(self):
        return [self.left, self.right]

    def cache_need(self):
        return None

    def cache_needs(self) -> dict:
        """name -> need of the mixers that want a cache or a state; the step's views come back under the same names."""
        needs = {}
        for side in self.SIDES:
            needs.update(side_needs(side, getattr(self, side)))
        return needs

    # what the two decide on the host per step is theirs: the decoder asks this part, which asks them
    def plan_step(self, step):
        for side in (self.left, self.right):
            if hasattr(side, "plan_step"):
                side.plan_step(step)

    def graph_key(self, step):
        return tuple(side.graph_key(step) for side in (self.left, self.right) if hasattr(side, "graph_key"))

    @property
    def plan_key(self):
        return (self.spec.kind, getattr(self.left, "plan_key", id(self.left)), getattr(self.right, "plan_key", id(self.right)))


@register_part("mixer", "side_by_side")
class SideBySide(Sides):
    """params: hidden_size, left (PartSpec), right (PartSpec), norm_eps, weight (0.5).
    tensors: left_out, right_out [hidden]."""
    native_libraries = ("norm_mix",)
    PARTIAL_FROM = 64                    # rows from which the mix kernel adds partial sums up itself

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.norm_eps = float(p["norm_eps"])
        self.weight = float(p.get("weight", 0.5))
        self.left = build_part("mixer", p["left"], ctx)
        self.right = build_part("mixer", p["right"], ctx)
        if getattr(self.left, "honours_partial_side", False):
            self.left.partial_side = True
        self.w_left = self.w_right = None

    def weight_shapes(self):
        return {"left_out": (self.hidden,), "right_out": (self.hidden,)}

    def load(self, tensors):
        self.w_left = tensors["left_out"].contiguous()
        self.w_right = tensors["right_out"].to(self.w_left.dtype).contiguous()

    def forward(self, h, out, step, cache):
        n = h.shape[0]
        dt = self.ctx.dtype
        ws = step.workspace
        results = []
        for side in self.SIDES:
            buf = ws.rows(f"side_{side}", n, self.hidden, dt)
            part = getattr(self, side)
            left = part.forward(h, buf, step, side_view(side, part, cache))
            if left is not None and (n < self.PARTIAL_FROM or
                                     (side == "left" and not getattr(part, "partial_side", False))):
                # a handful of rows: the reduce kernel's many blocks are faster than one block a row; a left mixer
                # that used the first scratch buffer: the right mixer's products would overwrite the sums
                left = left.reduce_into(buf)
            results.append(buf if left is None else left)
        ops.rms_mix(results[0], results[1], self.w_left, self.w_right, out, self.norm_eps, self.weight)
        return None


@register_part("mixer", "side_by_side_sum")
class SumSideBySide(Sides):
    """The layer's result is left_scale * left(h) + right_scale * right(h), without norms.

    Both are mixers between two products (`ProjectedMixer`), so the pair needs two products and not four: their input
    matrices are stacked along the outputs (both read h), their output matrices along the inputs (the sum of two
    products is the product of the operands side by side).  Each core writes its columns of the one operand, its
    scale applied before they are rounded.  (Zero rows between the two input matrices let the right mixer's columns start on
    a multiple of eight, for its wide loads.)
    params: hidden_size, left (PartSpec), right (PartSpec), left_scale, right_scale.  tensors: none of its own (it
    holds the children's matrices)."""

    honours_partial_side = True          # with `partial_side` set, the last product's partial sums go to the second scratch
    partial_side = False

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        tensors = {}
        for side in self.SIDES:
            part = build_part("mixer", p[side], ctx)
            if not isinstance(part, ProjectedMixer):
                raise ValueError(f"side_by_side_sum: {p[side].kind} is not a mixer between two products")
            part.joint = True
            part.result_scale = float(p[f"{side}_scale"])
            setattr(self, side, part)
            tensors.update({f"{side}.{slot}": p[side].tensors[slot] for slot in part.product_shapes()})
        self.spec = PartSpec(spec.kind, spec.params, tensors)
        self.right_at = -(-self.left.in_cols // 8) * 8
        self.in_cols = self.right_at + self.right.in_cols
        self.out_cols = self.left.out_cols + self.right.out_cols
        self.proj = self.o = None

    def weight_shapes(self):
        return {f"{side}.{slot}": shape for side in self.SIDES
                for slot, shape in getattr(self, side).product_shapes().items()}

    def load(self, tensors):
        mats = {side: [tensors[f"{side}.{slot}"] for slot in getattr(self, side).in_slots] for side in self.SIDES}
        gap = self.right_at - self.left.in_cols
        if gap:
            mats["left"].append(torch.zeros((gap, self.hidden), dtype=mats["left"][0].dtype, device=mats["left"][0].device))
        mats = mats["left"] + mats["right"]
        outs = [tensors[f"{side}.{getattr(self, side).out_slot}"] for side in self.SIDES]
        if len({m.dtype for m in mats}) != 1 or len({m.dtype for m in outs}) != 1:
            raise ValueError("side_by_side_sum: the stacked matrices must be stored in one dtype")
        self.proj = Linear(mats)
        self.o = Linear([torch.cat(outs, dim=1)])

    def reserve(self, limits):
        if self.proj is not None:
            self.proj.reserve(self.ctx.dtype, limits.max_tokens)
            self.o.reserve(self.ctx.dtype, limits.max_tokens, side=self.partial_side)

    def forward(self, h, out, step, cache):
        n, dt, ws = h.shape[0], self.ctx.dtype, step.workspace
        proj = ws.rows("sides_proj", n, self.in_cols, dt)
        self.proj.forward(h, proj)
        y = ws.rows("sides_y", n, self.out_cols, dt)
        at_out = 0
        for side, at_in in zip(self.SIDES, (0, self.right_at)):
            part = getattr(self, side)
            part.core(proj[:, at_in:at_in + part.in_cols], y[:, at_out:at_out + part.out_cols], step,
                      side_view(side, part, cache))
            at_out += part.out_cols
        return self.o.forward(y, out, defer=True, side=self.partial_side)
