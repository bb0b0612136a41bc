"""Decoder: a ModelPlan turned into parts, and the pass of one step through them.

The pass is the order list of the plan: embed the step's tokens into the
residual stream, run each entry's block against its cache, norm the rows whose
logits are wanted and project them to the vocabulary.  It is
fastllm_py/model.py:437-477 with three differences: it runs a flat batch of
tokens from many requests, it reads and writes the cache through the step's
tables, and it computes logits only at the wanted rows.
"""
from __future__ import annotations

import torch

from .base import BuildContext, ResidualStream
from .plan import ModelPlan
from .registry import build_part, part_class


class Decoder:
    def __init__(self, plan: ModelPlan, ctx: BuildContext):
        plan.validate()
        self.plan = plan
        self.ctx = ctx
        self.hidden = plan.hidden_size
        self.vocab = plan.vocab_size
        self.embedding = build_part("embedding", plan.embedding, ctx)
        self.blocks = [part_class("block", layer.block)(layer, ctx) for layer in plan.layers]
        self.final_norm = build_part("norm", plan.final_norm, ctx)
        self.head = build_part("head", plan.head, ctx)
        self.vectors = build_part("vectors", plan.vectors, ctx) if plan.vectors is not None else None
        self.entry = build_part("entry", plan.entry, ctx) if plan.entry is not None else None
        self.order = list(plan.order)
        # cache id of each run and, for a mixer with several needs, their names
        self._views_of = []
        for i, run in enumerate(self.order):
            mixer = self.blocks[run.layer].mixer
            names = tuple(mixer.cache_needs()) if hasattr(mixer, "cache_needs") else ()
            self._views_of.append((i if run.cache is None else run.cache, names))
        self.observer = None
        for i, run in enumerate(self.order):
            need = self.blocks[run.layer].mixer.cache_need()
            if run.cache is not None and need is not None:
                raise ValueError(f"order[{i}] reads run {run.cache}'s cache but its layer's mixer "
                                 f"wants a cache of its own")
            if run.cache is None and need is None and \
                    getattr(self.blocks[run.layer].mixer, "shares_cache", False):
                raise ValueError(f"order[{i}]: the layer shares a cache but the run names none")

    # ------------------------------------------------------------------ parts
    def all_parts(self):
        """Every part, nested ones included, each once."""
        out, seen = [], set()

        def visit(p):
            if id(p) in seen:
                return
            seen.add(id(p))
            out.append(p)
            for c in p.children():
                visit(c)

        visit(self.embedding)
        if self.vectors is not None:
            visit(self.vectors)
        if self.entry is not None:
            visit(self.entry)
        for b in self.blocks:
            visit(b)
        visit(self.final_norm)
        visit(self.head)
        return out

    def expected_tensors(self) -> dict:
        """checkpoint name -> shape, over all parts (a name shared by two parts once)."""
        table = {}
        for part in self.all_parts():
            spec = part.spec
            tensors = getattr(spec, "tensors", None)
            if tensors is None:
                continue
            shapes = part.weight_shapes()
            missing = set(shapes) - set(tensors)
            if missing:
                raise ValueError(f"{type(part).__name__}: the plan names no tensor for {sorted(missing)}")
            for slot, shape in shapes.items():
                name = tensors[slot]
                if name in table and tuple(table[name]) != tuple(shape):
                    raise ValueError(f"tensor {name} is wanted as {table[name]} and as {shape}")
                table[name] = tuple(shape)
        return table

    def load(self, tensors_by_name: dict) -> None:
        """Hands every part its tensors.  A part is told beforehand (`shared_slots`) which of its
        slots hold a tensor that another part holds too (a tied embedding table): it must leave
        such a tensor as it is."""
        users: dict = {}
        for part in self.all_parts():
            tensors = getattr(part.spec, "tensors", None)
            if tensors is not None:
                for slot in part.weight_shapes():
                    users[tensors[slot]] = users.get(tensors[slot], 0) + 1
        for part in self.all_parts():
            tensors = getattr(part.spec, "tensors", None)
            if tensors is None:
                continue
            shapes = part.weight_shapes()
            part.shared_slots = frozenset(slot for slot in shapes if users[tensors[slot]] > 1)
            part.load({slot: tensors_by_name[tensors[slot]] for slot in shapes})

    EMBEDDING_STATE = "embedding"        # cache id of the embedding part's per-request state

    def cache_needs(self) -> dict:
        """cache id -> need: the run index for the runs whose mixer owns a cache or a state; (run index, name) for
        each need of a mixer that has several (`cache_needs()`: mixers side by side); ("block", run index)
        for a block arrangement with per-request state of its own (`state_need()`); `EMBEDDING_STATE` for an
        embedding part with one."""
        needs = {}
        for i, run in enumerate(self.order):
            if run.cache is None:
                mixer = self.blocks[run.layer].mixer
                need = mixer.cache_need()
                if need is not None:
                    needs[i] = need
                for name, sub in (mixer.cache_needs() if hasattr(mixer, "cache_needs") else {}).items():
                    needs[(i, name)] = sub
            fn = getattr(self.blocks[run.layer], "state_need", None)
            need = fn() if fn is not None else None
            if need is not None:
                needs[("block", i)] = need
        fn = getattr(self.embedding, "state_need", None)
        need = fn() if fn is not None else None
        if need is not None:
            needs[self.EMBEDDING_STATE] = need
        return needs

    @property
    def graph_safe(self) -> bool:
        """False when some part says that its forward decides things on the host from the
        step's host copies (attribute `graph_safe = False`): its steps are never captured."""
        safe = getattr(self, "_graph_safe", None)
        if safe is None:                                    # (the parts are fixed once the decoder is built)
            safe = self._graph_safe = all(getattr(p, "graph_safe", True) for p in self.all_parts())
        return safe

    def _mixers_with(self, hook: str) -> list:
        """The mixers that have `hook`, one per `plan_key` (mixers of equal keys decide alike)."""
        cache = self.__dict__.setdefault("_hooked", {})
        if hook not in cache:
            found, seen = [], set()
            for block in self.blocks:
                mixer = block.mixer
                if not hasattr(mixer, hook):
                    continue
                key = getattr(mixer, "plan_key", None) or id(mixer)
                if key not in seen:
                    seen.add(key)
                    found.append(mixer)
            cache[hook] = found
        return cache[hook]

    def plan_step(self, step) -> None:
        """Before a step is launched: every mixer that decides something on the host for it
        (how to split the keys of a decode kernel, say) does so now and keeps it in `step.plans`."""
        for mixer in self._mixers_with("plan_step"):
            mixer.plan_step(step)

    def graph_key(self, step):
        """What, beside the number of tokens, fixes the launch shapes of a
        decode-only step: each mixer may add its own (a bucket of the longest
        sequence, say).  Steps with equal keys may replay one captured graph."""
        return tuple(mixer.graph_key(step) for mixer in self._mixers_with("graph_key"))

    @property
    def takes_fed_tokens(self) -> bool:
        """True when the embedding part can take a token from the sampler's output on the device."""
        return bool(getattr(self.embedding, "takes_fed_tokens", False))

    def reserve(self, limits, workspace) -> None:
        """Called once when an engine is built: every part sizes its scratch memory, and the
        buffers whose size follows the requests rather than the tokens get their steady size."""
        for part in self.all_parts():
            fn = getattr(part, "reserve", None)
            if fn is not None:
                fn(limits)
        rows = min(limits.max_tokens, limits.max_requests)
        workspace.rows("logits", rows, self.vocab, torch.float32, initial=rows)
        workspace.rows("picked", rows, self.hidden, self.ctx.dtype, initial=rows)

    # ------------------------------------------------------------------- pass
    def forward(self, step) -> torch.Tensor:
        """Logits [wanted rows, vocab] in float32 for the step's tokens."""
        n = step.n_tokens
        ws = step.workspace
        stream = ResidualStream(ws.rows("residual", n, self.hidden, torch.float32),
                                spill=lambda name="delta": ws.rows(name, n, self.hidden, self.ctx.dtype))
        if hasattr(self.embedding, "state_need"):
            self.embedding.forward(step, stream.x, step.cache_view(self.EMBEDDING_STATE, True))
        else:
            self.embedding.forward(step, stream.x)
        if self.entry is not None:
            self.entry.keep(stream, step)
        for i, run in enumerate(self.order):
            cache_id, names = self._views_of[i]
            block = self.blocks[run.layer]
            if names:                                          # several caches or states: the views by name
                cache = {name: step.cache_view((cache_id, name), run.cache is None) for name in names}
            else:
                cache = step.cache_view(cache_id, run.cache is None)
            if run.entry:
                self.entry.forward(stream, step)
            if run.vector is not None:
                stream.add_vector(self.vectors.row(run.vector))
            if hasattr(block, "state_need"):
                block.forward(stream, step, cache, step.cache_view(("block", i), True))
            else:
                block.forward(stream, step, cache)
            if self.observer is not None:                      # (a debugging aid: sees the stream after every run,
                self.observer(i, stream)                       # with the run's last sum (and bias) still pending)
        m = step.n_wanted
        logits = ws.rows("logits", m, self.vocab, torch.float32, initial=64)
        if m > 0:
            picked = ws.rows("picked", m, self.hidden, self.ctx.dtype, initial=64)
            rows = None if step.rows_identity else step.logit_rows
            stream.norm_into(self.final_norm, picked, rows=rows)
            self.head.forward(picked, logits)
        return logits
