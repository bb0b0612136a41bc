"""ModelPlan: a model written down as data.

An architecture's `make_plan(config, tensor_names)` returns one of these.  It
names, for every layer, which mixer, feed-forward, norms and position encoding
it has (kind + sizes + constants + the checkpoint names of its tensors), and in
which order the layers run.  The runtime (`parts.decoder.Decoder`) builds the
parts from the registries in `parts.registry` and never looks at the
architecture again.

fastllm-py derives the same information on the fly inside its one forward
function from the config and from which tensor names exist
(fastllm_py/model.py:399-470); a plan is that decision taken once, up front.
"""
from __future__ import annotations

from dataclasses import dataclass, field


@dataclass(frozen=True)
class PartSpec:
    """One part: `kind` selects the class, `params` are its sizes and constants
    (a nested PartSpec is allowed, e.g. a mixer's position encoding), `tensors`
    maps the part's own slot names to tensor names in the checkpoint."""
    kind: str
    params: dict = field(default_factory=dict)
    tensors: dict = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    """A layer = an arrangement (`block`) of a mixer, a feed-forward and norms.  An arrangement with sizes,
    constants or tensors of its own (a gate on the residual branch, say) has them in `params` and `tensors`."""
    block: str
    mixer: PartSpec
    feed_forward: PartSpec | None      # None: the layer is a mixer only (blocks that allow it)
    norms: dict            # role in the block -> PartSpec
    params: dict = field(default_factory=dict)
    tensors: dict = field(default_factory=dict)     # the block's own slots -> tensor names in the checkpoint


@dataclass(frozen=True)
class LayerRun:
    """One entry of the running order.

    `layer` indexes ModelPlan.layers; a layer may be named in several runs.
    `cache` names the cache (or state) this run uses: by default a cache of its
    own; the number of an earlier run to read that run's cache instead, in which
    case this run writes nothing to it.  `vector`: the row of ModelPlan.vectors that is
    added to the residual stream before this run (None: none).  `entry`: before that, the
    stream passes ModelPlan.entry."""
    layer: int
    cache: int | None = None
    vector: int | None = None
    entry: bool = False


@dataclass
class ModelPlan:
    hidden_size: int
    vocab_size: int
    max_positions: int
    embedding: PartSpec
    layers: list
    order: list
    final_norm: PartSpec
    head: PartSpec
    vectors: PartSpec | None = None      # a table [n, hidden] of vectors that runs start with (LayerRun.vector)
    entry: PartSpec | None = None        # what the stream passes before runs that say so (LayerRun.entry)
    ignorable: tuple = ()      # fnmatch patterns of checkpoint names that may be present and are not used

    def validate(self):
        n = len(self.layers)
        for i, run in enumerate(self.order):
            if not 0 <= run.layer < n:
                raise ValueError(f"order[{i}] names layer {run.layer}, plan has {n} layers")
            if run.vector is not None and self.vectors is None:
                raise ValueError(f"order[{i}] starts with vector {run.vector}, but the plan has no vectors")
            if run.entry and self.entry is None:
                raise ValueError(f"order[{i}] starts with the plan's entry, but the plan has none")
            if run.cache is not None:
                if not 0 <= run.cache < i:
                    raise ValueError(f"order[{i}] reads the cache of run {run.cache}, "
                                     f"which is not an earlier run")
                if self.order[run.cache].cache is not None:
                    raise ValueError(f"order[{i}] reads the cache of run {run.cache}, "
                                     f"which has no cache of its own")

    def tensor_names(self):
        """Every checkpoint tensor name the plan uses (a shared name once)."""
        names = []
        seen = set()

        def visit(spec):
            for name in spec.tensors.values():
                if name not in seen:
                    seen.add(name)
                    names.append(name)
            for v in spec.params.values():
                if isinstance(v, PartSpec):
                    visit(v)

        visit(self.embedding)
        if self.vectors is not None:
            visit(self.vectors)
        if self.entry is not None:
            visit(self.entry)
        for layer in self.layers:
            for name in layer.tensors.values():
                if name not in seen:
                    seen.add(name)
                    names.append(name)
            visit(layer.mixer)
            if layer.feed_forward is not None:
                visit(layer.feed_forward)
            for spec in layer.norms.values():
                visit(spec)
        visit(self.final_norm)
        visit(self.head)
        return names
