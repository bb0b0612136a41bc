"""Grouped-query softmax attention whose queries and keys are normed, head by head or over the whole projection.

Per token: q = W_q h (+ b_q), k = W_k h (+ b_k), v = W_v h (+ b_v), one stacked product; query head h reads
key/value head h // (heads / kv_heads); keys have `dim`, values `vdim` elements.  Each query and key head passes an
RMS norm over its `dim` elements: `qk_norm` "weighted" norms before the rotation with a weight [dim] that the heads
share, "unit" after the rotation without a weight; or, with "whole", all query heads of a token pass one RMS norm and all
key heads another, with a weight per column, before the rotation.  The rotation (a `position` part's tables) turns a head's first
`rot_dim` dimensions in pairs (2i, 2i + 1) (`pairing` "interleaved") or (i, i + rot_dim / 2) ("half").  With
`q_temp` = (coef, every) a query at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1).

    s_ij = q_i . k_j * scale;    p_ij = exp(s_ij) / ([exp(sink_head) +] sum over visible j' of exp(s_ij'))
    visible: j <= i, and with `window` w: i - j < w; with `chunk` c: floor(i / c) = floor(j / c)

The sink is one learned number per head in the denominator, without key or value; `sink` "unit" is a sink whose number
is 0 (one more unit in the denominator).  With `values_from_keys` there is no W_v: a token's value is its key as
projected, before norm and rotation.  With `head_gate` head h's result is multiplied by sigmoid(W_g h)_h, one number per
head and token; with `channel_gate` the concatenated heads by sigmoid(W_g h), one per channel (both in the attention
kernels, before they round).  W_g rides in the stacked product.  With `taps` every channel of q, k and v passes a causal
convolution over time, directly after the projection and its bias; a request's last taps - 1 projected rows are state
beside its cache.  With `out_bias` the output projection has a bias, which a block that can adds with the pending sum.

The attention itself is the sink-attention kernels' (CUDA cores in 32-bit; tensor cores for prompt portions and
split keys for single tokens in bfloat16), which take the chunk beside the window.
"""
from __future__ import annotations

import torch

from ..cache.needs import FixedState, PagedKeysValues
from ..native import ops, scratch
from .base import ProjectedMixer
from .registry import build_part, register_part


@register_part("mixer", "normed_attention")
class NormedAttention(ProjectedMixer):
    """params: hidden_size, heads, kv_heads, dim, vdim, scale, norm_eps, qk_norm (None | "weighted" | "unit" |
    "whole"),
    position (PartSpec | None), pairing ("half" | "interleaved"), q_temp (None | (coef, every)), window (None | int),
    chunk (None | int), sink (False | True | "unit"), biases (bool), out_bias (bool), taps (None: no convolution),
    values_from_keys (bool), head_gate (bool), channel_gate (bool).
    tensors: q [heads * dim, hidden], k [kv_heads * dim, hidden], o [hidden, heads * vdim]; v [kv_heads * vdim, hidden]
    unless values_from_keys; with biases q_bias, k_bias (and v_bias); with out_bias o_bias [hidden]; for "weighted"
    q_norm, k_norm [dim], for "whole" [heads * dim], [kv_heads * dim]; with taps q_conv, k_conv, v_conv [channels, taps]; with sink True sink [heads]; with a gate
    gate [heads, hidden] or [heads * vdim, hidden]."""
    category = "mixer"
    SCRATCH = "sink attention splits"
    workspace_name = "normed_attention"
    out_bias = None                      # float32 [hidden] where the output projection has one
    defers_out_bias = False              # set by a block that adds `out_bias` itself, with the pending sum

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.heads, self.kv_heads = int(p["heads"]), int(p["kv_heads"])
        self.dim, self.vdim = int(p["dim"]), int(p["vdim"])
        self.scale = float(p["scale"])
        self.norm_eps = float(p.get("norm_eps", 1e-6))
        self.qk_norm = p.get("qk_norm")
        self.pairing = p.get("pairing", "half")
        self.q_temp = tuple(p["q_temp"]) if p.get("q_temp") else None
        self.window = int(p["window"]) if p.get("window") else None
        self.chunk = int(p["chunk"]) if p.get("chunk") else None
        self.sink_kind = p.get("sink", False)
        self.biases = bool(p.get("biases", False))
        self.has_out_bias = bool(p.get("out_bias", False))
        self.taps = int(p["taps"]) if p.get("taps") is not None else None
        self.back = self.taps - 1 if self.taps else 0         # rows of a sequence that the convolution keeps
        self.v_from_k = bool(p.get("values_from_keys", False))
        self.gated = bool(p.get("head_gate", False))
        self.channel_gated = bool(p.get("channel_gate", False))
        if self.heads % self.kv_heads:
            raise ValueError(f"normed_attention: {self.heads} heads are not a multiple of {self.kv_heads} kv heads")
        if self.qk_norm not in (None, "weighted", "unit", "whole"):
            raise ValueError(f"normed_attention: qk_norm {self.qk_norm!r} is none of None, 'weighted', 'unit', 'whole'")
        if self.qk_norm == "whole" and (self.taps is not None or self.v_from_k or self.q_temp):
            raise ValueError("normed_attention: norms over the whole projection do not go with a convolution, keys as values "
                             "or scaled queries")
        if self.pairing not in ("half", "interleaved"):
            raise ValueError(f"normed_attention: pairing {self.pairing!r} is neither 'half' nor 'interleaved'")
        if self.sink_kind not in (False, True, "unit"):
            raise ValueError(f"normed_attention: sink {self.sink_kind!r} is none of False, True, 'unit'")
        if self.v_from_k and self.vdim != self.dim:
            raise ValueError("normed_attention: keys that serve as values have the values' size")
        if self.vdim > 256:
            raise ValueError(f"normed_attention: value size {self.vdim} is beyond the kernels' limit of 256")
        if self.v_from_k and self.taps:
            raise ValueError("normed_attention: a convolution does not go with keys that serve as values")
        if self.gated and self.channel_gated:
            raise ValueError("normed_attention: a gate per head or one per channel, not both")
        self.position = build_part("position", p["position"], ctx) if p.get("position") else None
        if self.position is not None and self.position.rot_dim > self.dim:
            raise ValueError("normed_attention: the position encoding turns more dimensions than a head has")
        self.q_cols, self.k_cols = self.heads * self.dim, self.kv_heads * self.dim
        self.v_cols = 0 if self.v_from_k else self.kv_heads * self.vdim
        self.channels = self.q_cols + self.k_cols + self.v_cols
        self.gate_cols = self.heads if self.gated else self.heads * self.vdim if self.channel_gated else 0
        self.in_cols, self.out_cols = self.channels + self.gate_cols, self.heads * self.vdim
        self.in_slots = ("q", "k") + (() if self.v_from_k else ("v",)) + (("gate",) if self.gate_cols else ())
        self.bias = self.q_w = self.k_w = self.sink = self.conv_w = None

    @property
    def native_libraries(self):
        return ("sink_attention", "conv_head") if self._conv_prep() else ("sink_attention",)

    def _conv_prep(self) -> bool:
        """Whether the preparation with a convolution (or a factor on the values) serves this part."""
        return (self.taps is not None or self.joint) and not self.v_from_k and self.qk_norm != "whole"

    def children(self):
        return [self.position] if self.position is not None else []

    def _cache(self):
        # behind a chunk's start nothing is seen again: at most `chunk` tokens back, like a window of that size
        reach = min(x for x in (self.window, self.chunk) if x) if (self.window or self.chunk) else None
        return PagedKeysValues(self.kv_heads, self.dim, self.vdim, reach, 0)

    def cache_need(self):
        return self._cache() if self.back == 0 else None

    def cache_needs(self) -> dict:
        """With a convolution: the keys and values, and the last projected rows."""
        if self.back == 0:
            return {}
        return {"kv": self._cache(), "conv": FixedState((self.back * self.channels,), "float32")}

    def in_rows(self):
        rows = {"q": self.q_cols, "k": self.k_cols, "v": self.v_cols, "gate": self.gate_cols}
        return {slot: rows[slot] for slot in self.in_slots}

    def core_shapes(self):
        shapes = {}
        cols = {"q": self.q_cols, "k": self.k_cols, **({} if self.v_from_k else {"v": self.v_cols})}
        if self.biases:
            shapes.update({f"{s}_bias": (n,) for s, n in cols.items()})
        if self.has_out_bias:
            shapes["o_bias"] = (self.hidden,)
        if self.qk_norm == "weighted":
            shapes.update({"q_norm": (self.dim,), "k_norm": (self.dim,)})
        elif self.qk_norm == "whole":
            shapes.update({"q_norm": (self.q_cols,), "k_norm": (self.k_cols,)})
        if self.taps:
            shapes.update({f"{s}_conv": (n, self.taps) for s, n in cols.items()})
        if self.sink_kind is True:
            shapes["sink"] = (self.heads,)
        return shapes

    def load_core(self, tensors):
        cols = ["q", "k"] + ([] if self.v_from_k else ["v"])
        if self.joint and (self.has_out_bias or self.v_from_k):
            raise ValueError("normed_attention: an output bias, or keys as values, do not go with shared products")
        if self.result_scale != 1.0 and not self._conv_prep() and self.qk_norm != "whole":
            raise ValueError("normed_attention: a factor on the result needs values of their own")
        if self.biases:
            self.bias = torch.cat([tensors[f"{s}_bias"].float() for s in cols]).contiguous()
        if self.has_out_bias:
            self.out_bias = tensors["o_bias"].float().clone()
        if self.qk_norm in ("weighted", "whole"):
            self.q_w = tensors["q_norm"].float().contiguous()
            self.k_w = tensors["k_norm"].float().contiguous()
        if self.taps:                                         # [taps, channels]: the kernel reads along the channels
            self.conv_w = torch.cat([tensors[f"{s}_conv"].float() for s in cols]).t().contiguous()
        if self.sink_kind is True:
            self.sink = tensors["sink"].float().contiguous()
        elif self.sink_kind == "unit":
            self.sink = torch.zeros(self.heads, dtype=torch.float32, device=self.ctx.device)

    def _tc(self) -> bool:
        return self.ctx.device.type == "cuda" and ops.sink_tc_takes(self.ctx.dtype, self.dim, self.vdim)

    def native_builds(self):
        """(library, defines) pairs compiled for this part's sizes, so that a model's first load builds them beside
        its other libraries."""
        return [ops.sink_tc_library(self.dim, self.vdim)] if self._tc() else []

    def reserve(self, limits):
        super().reserve(limits)
        if self._tc():
            from ..native.build import load_library
            load_library(*ops.sink_tc_library(self.dim, self.vdim))        # built now, not inside the first step
        if self.ctx.device.type == "cuda" and self._splits_single_tokens():
            longest = -(-limits.max_model_len // 1024) * 1024
            self._partials(min(limits.max_tokens, limits.max_requests),
                           ops.sink_decode_splits(self.window, 0, longest, self.chunk)[0])   # nothing grows under a graph

    # ---- what the host decides per step: how many blocks share a single token's keys
    @property
    def plan_key(self):
        return ("normed_attention", self.heads, self.kv_heads, self.dim, self.vdim, self.window, self.chunk)

    def _splits_single_tokens(self) -> bool:
        """bfloat16 steps give their single tokens to the split-key kernels (the 32-bit path keeps one kernel for every
        token, so that its sums do not depend on how a sequence was cut)."""
        return self.ctx.dtype == torch.bfloat16 and ops.sink_decode_takes(self.heads, self.kv_heads, self.dim, self.vdim)

    def plan_step(self, step):
        if not self._splits_single_tokens() or step.n_decode_tokens == 0:
            step.plans[self.plan_key] = (1, 0)
            return
        longest = step.max_seq_len
        if step.for_graph:                                    # a captured step serves many: cover the length rounded up
            longest = -(-longest // 1024) * 1024
        step.plans[self.plan_key] = ops.sink_decode_splits(self.window, 0, longest, self.chunk)

    def graph_key(self, step):
        return step.plans.get(self.plan_key)

    def _partials(self, n_tokens: int, n_splits: int):
        return scratch.get(self.ctx.device, self.SCRATCH, n_tokens * self.heads * n_splits * (self.vdim + 2))

    def _prepare(self, proj, q, step, cache, tail):
        """Queries to `q`, keys and values to the tokens' cache rows."""
        cos, sin = self.position.tables() if self.position is not None else (None, None)
        rot = self.position.rot_dim if self.position is not None else 0
        mode = {"weighted": 1, "unit": 2}.get(self.qk_norm, 0)
        interleaved = self.pairing == "interleaved"
        if self.qk_norm == "whole":
            ops.sink_prep(proj, self.bias, self.q_w, self.k_w, self.norm_eps, q, self.heads, self.kv_heads, self.dim, self.vdim, 0,
                          0.0, None, cache.slots, cache.tensor, cache.page_size, rot, interleaved, cos, sin, step.positions,
                          self.result_scale)
        elif self._conv_prep():
            ops.conv_head_prep(proj, self.bias, self.conv_w, tail, self.q_w, self.k_w, mode, self.norm_eps, rot, interleaved, cos,
                               sin, step, self.q_temp, self.result_scale, q, self.heads, self.kv_heads, self.dim, self.vdim,
                               cache.slots, cache.tensor, cache.page_size)
        else:
            ops.head_prep(proj, self.bias, self.q_w, self.k_w, mode, self.norm_eps, rot, interleaved, cos, sin, step.positions,
                          self.q_temp, self.v_from_k, q, self.heads, self.kv_heads, self.dim, self.vdim, cache.slots,
                          cache.tensor, cache.page_size)

    def core(self, proj, ctx, step, cache):
        n = proj.shape[0]
        dt = self.ctx.dtype
        tail = None
        if self.back:
            tail, cache = cache["conv"].tensor, cache["kv"]
        q = step.workspace.rows("normed_attention_q", n, self.q_cols, dt)
        self._prepare(proj, q, step, cache, tail)
        gate = proj[:, self.channels:self.channels + self.gate_cols] if self.gate_cols else None
        tc = self._tc()
        # (where only the CUDA-core kernel serves prompt rows, a mixed step gives it every row)
        single = step.n_decode_tokens if self._splits_single_tokens() and (tc or step.n_decode_tokens == n) else 0
        if single:                                            # single tokens: their keys split over blocks
            if self.plan_key not in step.plans:               # a step built by hand, not by the engine
                self.plan_step(step)
            n_splits, kept_splits = step.plans[self.plan_key]
            ops.sink_decode(q, ctx, cache.tensor, cache.block_table, step.tok_req, step.positions, step.decode_tokens,
                            self._partials(single, n_splits), n_splits, kept_splits, self.heads, self.kv_heads,
                            self.dim, self.vdim, self.window, 0, self.scale, None, None, None, self.sink, cache.page_size,
                            chunk=self.chunk, gate=gate)
        if single == n:
            pass
        elif tc:
            ops.sink_attention_tc(q, ctx, cache.tensor, cache.block_table, step, self.heads, self.kv_heads, self.dim,
                                  self.vdim, self.window, 0, self.scale, None, None, None, self.sink, cache.page_size,
                                  include_single=not single, chunk=self.chunk, gate=gate)
        else:
            ops.sink_attention_simt(q, ctx, cache.tensor, cache.block_table, step.tok_req, step.positions, self.heads,
                                    self.kv_heads, self.dim, self.vdim, self.window, 0, self.scale, None, None, None,
                                    self.sink, cache.page_size, chunk=self.chunk, gate=gate)

    def forward(self, h, out, step, cache):
        left = super().forward(h, out, step, cache)
        if self.out_bias is None or self.defers_out_bias:
            return left
        if left is not None:
            left.reduce_into(out)
        ops.add_bias(out, self.out_bias)
        return None
