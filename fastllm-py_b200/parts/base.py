"""What every part is, and what a part may ask of the engine while it runs.

A part is built from a PartSpec (kind, sizes and constants, tensor names) and a
BuildContext (device, activation dtype, page size).  It declares the shapes of
its tensors by slot, receives them at load, and runs on the tokens of one step.
It knows nothing of the model it is in: names of checkpoint tensors, the number
of layers and the architecture stay in the plan.

Interfaces by category (all tensors are torch CUDA tensors; `step` is the
engine's StepContext; buffers come from `step.workspace`):

  embedding     forward(step, out)            out: [N, hidden] float32 residual stream
  position      tables(max_positions)         -> (cos, sin) float32 [max_positions, rot_dim/2]
  norm          apply(stream, out, rows=None) adds the stream's pending sum, then norms into `out`
  mixer         cache_need() -> a need of cache.needs (paged, fixed state) | None
                forward(h, out, step, cache)  h: [N, hidden] -> out: [N, hidden]
  feed_forward  forward(h, out, step)
  block         forward(stream, step, cache)  the arrangement of mixer, feed-forward and norms
  head          forward(h, out)               h: [m, hidden] -> out: [m, vocab] float32
  entry         keep(stream, step)            the stream as the embedding leaves it
                forward(stream, step)         replaces the stream before a run of a layer

What a part may declare beside its interface (all optional; absent means "no"):

  reserve(limits)          any part: called once when an engine is built, with the most tokens
                           of a step, the most live requests and the longest sequence, so that
                           the part can size the scratch memory its kernels take
  plan_step(step)          mixer: called once per step before anything is launched; decides on
                           the host what the step's launches need (a split of the keys, say) and
                           keeps it in `step.plans`; mixers with an equal `plan_key` are asked once
  graph_key(step)          mixer: what of that plan fixes the launch shapes (part of the key
                           under which a captured step is replayed)
  graph_safe = False       any part whose forward decides on the host from the step's host copies
  takes_partial = True     norm: `apply` accepts split-K partial sums as the stream's pending sum
                           (otherwise the stream adds them up into a tensor first)
  takes_post_norm = True   norm: `apply` understands `stream.pending_norm` (the pending sum is normed by
                           that part before it is added); such a norm also has `add_normed(stream)`
  takes_extra = True       norm: `apply` adds `stream.extra` (a second sum) along with the pending one, each a tensor
                           or partial sums, also under gathered rows, and row vectors where nothing is pending; such a
                           norm also has `apply_pair(stream, other, out, out_other)`: its own norm and that of
                           `other` (same kind, size and eps) of the one row in one pass
  takes_vectors = True     norm: `apply` adds `stream.vectors` (row vectors) along with a pending sum
  takes_fed_tokens = True  embedding: understands a token id -1 - r as "row r of `step.token_feed`"
                           (without it the scheduler never launches a step ahead of the host)
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch


@dataclass(frozen=True)
class EngineLimits:
    """The bounds an engine was built with, as parts see them in `reserve`."""
    max_tokens: int          # tokens of one step
    max_requests: int        # live requests (and so requests of one step)
    max_model_len: int       # longest sequence


@dataclass
class BuildContext:
    device: torch.device
    dtype: torch.dtype                 # activation / cache dtype: torch.bfloat16 or torch.float32
    page_size: int
    max_positions: int                 # position tables cover [0, max_positions)
    shared: dict = field(default_factory=dict)   # objects parts may share (position tables by spec)


class Part:
    category = None

    def __init__(self, spec, ctx: BuildContext):
        self.spec = spec
        self.ctx = ctx

    def weight_shapes(self) -> dict:
        """slot -> expected shape of the checkpoint tensor."""
        return {}

    shared_slots: frozenset = frozenset()    # set by the decoder before `load`: slots whose tensor another part holds too

    def load(self, tensors: dict) -> None:
        """Receives slot -> device tensor in its stored dtype.  A tensor of a slot in
        `shared_slots` belongs to another part as well and must be left as it is."""

    def children(self) -> list:
        """Parts nested inside this one (their tensors are loaded too)."""
        return []

    def reserve(self, limits: EngineLimits) -> None:
        """Size whatever scratch memory this part's kernels take for steps within `limits`."""


class ResidualStream:
    """The residual sum, float32 in both precisions, plus a sum not yet added.

    A mixer or feed-forward leaves its output as `pending`; the next norm adds
    it while it norms (one pass over the row instead of two), which is the
    deferred add of fastllm_py/graph_decode.py:810-813.  The pending sum is a
    tensor [N, hidden], or the split-K partial sums of the product that made it
    (an object with `reduce_into(tensor)`): a norm that says `takes_partial`
    adds the slabs while it reads, any other gets them added up first, into the
    buffer that `spill()` returns."""

    def __init__(self, x: torch.Tensor, spill=None):
        self.x = x
        self.pending = None
        self.pending_norm = None     # a norm part the pending sum passes before it is added (blocks that norm
        self.spill = spill           # a sublayer's output); a norm with `takes_post_norm` does both in one kernel
        self.extra = None            # a second sum not yet added (a layer whose mixer and feed-forward run side by
                                     # side leaves two; a tensor, or partial sums); a norm with `takes_extra` adds both while it reads
        self.pending_scale = 1.0     # the pending sum is multiplied by this as it is added (a layer that scales its
                                     # sublayers' results); a norm with `takes_scale` does so while it reads
        self.vectors = ()            # float32 row vectors [hidden] not yet added, each to every row (a product's output
                                     # bias, the vector that a pass of layers starts with)

    def add_vector(self, vector):
        """Every row is to be increased by `vector`, at the latest when the next norm reads the stream."""
        if len(self.vectors) == 2:
            self._add_vectors()
        self.vectors = self.vectors + (vector,)

    def _add_vectors(self):
        """x += the row vectors, for whoever cannot take them itself."""
        from ..native import ops
        ops.row_add(self.x, self.vectors)
        self.vectors = ()

    def _add_scaled(self):
        """x += pending_scale * pending (a tensor), for whoever cannot take the scale itself."""
        from ..native import ops
        ops.scaled_add(self.x, self.pending, self.pending_scale)
        self.pending, self.pending_scale = None, 1.0

    def settle(self):
        """x takes in whatever is still pending (for a block whose sublayers read x itself)."""
        from ..native import ops
        if self.vectors:
            self._add_vectors()
        if self.pending is not None and not isinstance(self.pending, torch.Tensor):
            self.pending = self.pending.reduce_into(self.spill())
        if self.pending is not None and self.pending_scale != 1.0:
            self._add_scaled()
        if self.pending is not None:
            if self.pending_norm is not None:
                self.pending_norm.add_normed(self)
            else:
                ops.residual_add(self.x, self.pending)
                self.pending = None
        self._add_extra()

    def _add_extra(self):
        """x += extra, for whoever cannot take it itself."""
        from ..native import ops
        if self.extra is not None:
            if not isinstance(self.extra, torch.Tensor):
                self.extra = self.extra.reduce_into(self.spill("delta_ff"))
            ops.residual_add(self.x, self.extra)
            self.extra = None

    def norm_into(self, norm, out, rows=None):
        """`norm.apply(self, out, rows)`, with a pending sum that the norm can take."""
        pending = self.pending
        if getattr(norm, "takes_extra", False) and self.pending_scale == 1.0 and self.pending_norm is None and \
                (self.extra is not None or (self.vectors and pending is None)):
            norm.apply(self, out, rows)                  # everything that waits is added while the row is read
            return
        if self.vectors and (pending is None or self.pending_scale != 1.0 or self.pending_norm is not None or
                             self.extra is not None or not getattr(norm, "takes_vectors", False)):
            self._add_vectors()
        if pending is not None and not isinstance(pending, torch.Tensor):
            both = getattr(norm, "takes_partial", False) and \
                (self.pending_scale == 1.0 or getattr(norm, "takes_scale", False)) and \
                (self.pending_norm is None or getattr(norm, "takes_post_norm", False))
            if rows is not None or not both:
                pending = self.pending = pending.reduce_into(self.spill())
        if pending is not None and self.pending_scale != 1.0 and not getattr(norm, "takes_scale", False):
            self._add_scaled()                           # (every row, also when only some are normed)
            pending = None
        if pending is not None and self.pending_norm is not None and not getattr(norm, "takes_post_norm", False):
            self.pending_norm.add_normed(self)           # x += norm(pending), for a norm that cannot do it itself
        self._add_extra()
        norm.apply(self, out, rows)


class Workspace:
    """Named activation buffers, made once for the most tokens a step may have.

    `rows(name, n, cols, dtype)` returns the first n rows of the buffer of that
    name; parts that run one after another share buffers by using the same
    name.  Row pitch is rounded up to 16 bytes (what a TMA descriptor wants)."""

    def __init__(self, device, max_tokens: int):
        self.device = device
        self.max_tokens = max_tokens
        self._buffers: dict = {}
        self._views: dict = {}           # (name, cols, dtype, n) -> the view handed out for it before
        self.generation = 0              # bumped when a buffer is replaced by a larger one

    def rows(self, name: str, n: int, cols: int, dtype, initial: int | None = None,
             first: int | None = None) -> torch.Tensor:
        """`initial` (for buffers that are wide but usually short, like logits)
        starts the buffer at that many rows and lets it grow to max_tokens on demand.
        `first`: only the first so many of the `cols` columns (the same memory as the
        whole rows: the queries of a q|k|v buffer, say)."""
        if first is not None:
            view = self._views.get((name, cols, dtype, n, first))
            if view is None:
                whole = self.rows(name, n, cols, dtype, initial)
                view = self._views[(name, cols, dtype, n, first)] = whole[:, :first]
            return view
        view = self._views.get((name, cols, dtype, n))
        if view is not None:             # (making a view costs a few microseconds: a step asks a hundred times)
            return view
        key = (name, cols, dtype)
        buf = self._buffers.get(key)
        if n > self.max_tokens:
            raise RuntimeError(f"a step of {n} rows exceeds the workspace's {self.max_tokens}")
        if buf is None or buf.shape[0] < n:
            if torch.cuda.is_available() and torch.cuda.is_current_stream_capturing():
                raise RuntimeError(f"workspace buffer {key} would be allocated during graph capture")
            unit = 16 // torch.empty((), dtype=dtype).element_size()
            pitch = -(-cols // unit) * unit
            cap = self.max_tokens if initial is None else min(self.max_tokens, max(initial, n))
            if buf is not None:
                cap = min(self.max_tokens, max(n, 2 * buf.shape[0]))
                self.generation += 1     # captured graphs may hold the old buffer's address
            buf = torch.zeros((cap, pitch), dtype=dtype, device=self.device)
            self._buffers[key] = buf
            for k in [k for k in self._views if k[:3] == key]:
                del self._views[k]
        if len(self._views) > 4096:
            self._views.clear()
        view = self._views[(name, cols, dtype, n)] = buf[:n, :cols]
        return view


class ProjectedMixer(Part):
    """A mixer between two matrix products: one stacked product of the input, a core that turns a token's columns of it
    (with a cache or state) into the operand of the second, and that second product.

    A subclass names the matrices (`in_slots`, stacked in this order; `out_slot`), their widths (`in_cols`, `out_cols`,
    `hidden`), the other tensors (`core_shapes`, `load_core`) and the core itself:

        core(proj, y, step, cache)    proj [N, in_cols] -> y [N, out_cols]

    Two such mixers that read the same input can share both products (`side_by_side_sum`): the parent sets `joint` before
    the tensors are loaded, holds the matrices itself and calls the cores.  `result_scale` is a factor on the mixer's
    result that the core applies where it costs nothing (before y is rounded)."""
    joint = False
    result_scale = 1.0
    in_slots: tuple = ()
    out_slot = "o"
    in_cols = out_cols = hidden = 0
    workspace_name = "mixer"
    honours_partial_side = True          # with `partial_side` set, the last product's partial sums go to the second scratch
    partial_side = False
    proj = o = None

    def in_rows(self) -> dict:
        """slot -> rows of its matrix."""
        raise NotImplementedError

    def core_shapes(self) -> dict:
        return {}

    def product_shapes(self) -> dict:
        shapes = {slot: (rows, self.hidden) for slot, rows in self.in_rows().items()}
        shapes[self.out_slot] = (self.hidden, self.out_cols)
        return shapes

    def weight_shapes(self):
        return self.core_shapes() if self.joint else {**self.product_shapes(), **self.core_shapes()}

    def load_core(self, tensors) -> None:
        pass

    def load(self, tensors):
        from .linear import Linear
        if not self.joint:
            mats = [tensors[slot] for slot in self.in_slots]
            if len({m.dtype for m in mats}) != 1:
                raise ValueError(f"{self.workspace_name}: the stacked matrices must be stored in one dtype")
            self.proj = Linear(mats)
            self.o = Linear([tensors[self.out_slot]])
        self.load_core(tensors)

    def reserve(self, limits):
        if self.proj is not None:
            self.proj.reserve(self.ctx.dtype, limits.max_tokens)
            self.o.reserve(self.ctx.dtype, limits.max_tokens, side=self.partial_side)

    def core(self, proj, y, step, cache) -> None:
        raise NotImplementedError

    def forward(self, h, out, step, cache):
        n, dt, ws = h.shape[0], self.ctx.dtype, step.workspace
        proj = ws.rows(self.workspace_name + "_proj", n, self.in_cols, dt)
        self.proj.forward(h, proj)
        y = ws.rows(self.workspace_name + "_y", n, self.out_cols, dt)
        self.core(proj, y, step, cache)
        return self.o.forward(y, out, defer=True, side=self.partial_side)
