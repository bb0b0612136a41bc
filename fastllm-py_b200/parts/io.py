"""Embedding and output head.

Embedding: x = table[ids] (fastllm_py/model.py:447), times `scale` for designs that scale it.  Head:
logits = x @ W^T in float, no bias (model.py:476), then, for a head with a
`softcap` c, logits <- c * tanh(logits / c); with tied
embeddings the head's matrix is the embedding table itself (model.py:228-231),
which the loader expresses by giving both parts the same tensor."""
from __future__ import annotations

from ..native import ops
from .base import Part
from .linear import Linear
from .registry import register_part


@register_part("embedding", "table")
class Embedding(Part):
    """params: vocab_size, hidden_size, scale (1: none), norm_eps (None: the rows are not normed), norm_offset (0).
    tensors: weight [vocab, hidden]; with norm_eps norm [hidden]: the residual stream starts as the row divided by its
    root mean square times (norm_offset + norm)."""
    category = "embedding"
    takes_fed_tokens = True              # an id -1 - r is taken from row r of step.token_feed

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.vocab = int(spec.params["vocab_size"])
        self.hidden = int(spec.params["hidden_size"])
        self.scale = float(spec.params.get("scale", 1.0))
        self.norm_eps = spec.params.get("norm_eps")
        self.norm_offset = float(spec.params.get("norm_offset", 0.0))
        self.table = self.norm_w = None

    def weight_shapes(self):
        shapes = {"weight": (self.vocab, self.hidden)}
        if self.norm_eps is not None:
            shapes["norm"] = (self.hidden,)
        return shapes

    def load(self, tensors):
        self.table = tensors["weight"]
        if self.norm_eps is not None:
            self.norm_w = (tensors["norm"].double() + self.norm_offset).float().contiguous()

    def forward(self, step, out):
        ops.embed(self.table, step.token_ids, out, step.status, getattr(step, "token_feed", None), self.scale)
        if self.norm_w is not None:
            ops.rmsnorm(out, self.norm_w, out, self.norm_eps)       # in place: a thread rewrites what it read


@register_part("embedding", "table_pairs")
class PairEmbedding(Embedding):
    """x = table[id] * scale + pairs[(previous id * mul_prev + id * mul_cur) mod buckets]: a second, hashed table
    indexed by the token and the one before it; a sequence's first token takes the table's last row (`buckets`).
    The token before a step's first one is per-request state (one int32 per request slot).
    params: vocab_size, hidden_size, scale, norm_eps, norm_offset (as above; the sum is normed), buckets, mul_prev,
    mul_cur.  tensors: weight [vocab, hidden], pairs [buckets + 1, hidden], norm."""
    native_libraries = ("gated_block",)

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.buckets = int(spec.params["buckets"])
        self.mul_prev = int(spec.params["mul_prev"])
        self.mul_cur = int(spec.params["mul_cur"])
        if self.buckets < 1:
            raise ValueError("table_pairs: buckets must be at least 1")
        self.pairs = None

    def weight_shapes(self):
        return {**super().weight_shapes(), "pairs": (self.buckets + 1, self.hidden)}

    def state_need(self):
        from ..cache.needs import FixedState
        return FixedState((1,), "int32")

    def load(self, tensors):
        super().load(tensors)
        self.pairs = tensors["pairs"]
        if self.pairs.dtype != self.table.dtype:
            raise ValueError("table_pairs: both tables must be stored in one dtype")

    def forward(self, step, out, state):
        ops.pair_embed(self.table, self.pairs, out, step, state.tensor, self.buckets, self.mul_prev, self.mul_cur,
                       self.scale, self.norm_w, self.norm_eps or 0.0)


@register_part("vectors", "table")
class VectorTable(Part):
    """Vectors [n, hidden] that runs of layers start with: added to every row of the residual stream.
    params: count, hidden_size.  tensors: rows [count, hidden]."""
    category = "vectors"

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.count = int(spec.params["count"])
        self.hidden = int(spec.params["hidden_size"])
        self.table = None

    def weight_shapes(self):
        return {"rows": (self.count, self.hidden)}

    def load(self, tensors):
        # one allocation a row: every row starts on an aligned address, whatever the width
        self.table = [row.contiguous().clone() for row in tensors["rows"].float()]

    def row(self, i):
        return self.table[i]


@register_part("entry", "rejoin")
class Rejoin(Part):
    """x <- W [x; x0]: the residual stream replaced by a product of itself beside the embedding output.
    params: hidden_size.  tensors: weight [hidden, 2 hidden] (x first)."""
    category = "entry"

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.hidden = int(spec.params["hidden_size"])
        self.linear = None

    def weight_shapes(self):
        return {"weight": (self.hidden, 2 * self.hidden)}

    def load(self, tensors):
        self.linear = Linear([tensors["weight"]])

    def reserve(self, limits):
        if self.linear is not None:
            self.linear.reserve(self.ctx.dtype, limits.max_tokens)

    def _operand(self, stream, step):
        return step.workspace.rows("entry_operand", stream.x.shape[0], 2 * self.hidden, self.ctx.dtype)

    def keep(self, stream, step):
        ops.sum_rows(stream.x, None, None, self._operand(stream, step)[:, self.hidden:])

    def forward(self, stream, step):
        operand = self._operand(stream, step)
        if stream.pending_scale != 1.0 or stream.pending_norm is not None:
            stream.settle()
        ops.sum_rows(stream.x, stream.pending, stream.extra, operand[:, :self.hidden], stream.vectors)
        stream.pending = stream.extra = None
        stream.vectors = ()
        self.linear.forward(operand, stream.x)               # (float accumulation, float result)


@register_part("head", "linear")
class LinearHead(Part):
    """params: vocab_size, hidden_size, softcap (None | c > 0).  tensors: weight [vocab, hidden]."""
    category = "head"

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.vocab = int(spec.params["vocab_size"])
        self.hidden = int(spec.params["hidden_size"])
        self.softcap = spec.params.get("softcap")
        self.linear = None

    def weight_shapes(self):
        return {"weight": (self.vocab, self.hidden)}

    def load(self, tensors):
        # a table that the embedding part reads too stays row-major; a matrix of its own may be packed
        w = tensors["weight"]
        self.linear = Linear.sharing(w) if "weight" in self.shared_slots else Linear([w])

    def reserve(self, limits):
        if self.linear is not None:
            self.linear.reserve(self.ctx.dtype, min(limits.max_tokens, limits.max_requests))

    def forward(self, h, out):
        self.linear.forward(h, out)
        if self.softcap:
            ops.softcap(out, self.softcap)
