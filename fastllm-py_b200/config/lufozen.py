"""LufozenConfig: the typed configuration of the Lufozen decoder.

A Lufozen model is a list of pre-norm layers (RMS norms whose weights are stored around zero), some of which run
several times in a row with the same weights.  Its config.json is nested:

    architecture     "Lufozen"
    vocab, width     sizes of the embedding table and the residual stream
    norm.eps         the epsilon of every norm
    embedding        {"scale": s (absent: 1), "bigram": {"buckets", "mul_prev", "mul_cur"}}   (bigram absent: one table)
    loop             {"start", "stop", "times"}: layers start .. stop - 1 run `times` times in a row (absent: every layer
                     runs once); a stored vector per pass is added to the stream as the pass starts
    logit_scale      factor on the logits (absent: 1)
    layers[i]        {"type": "parallel" | "gla" | "attention", "mixer": {...}, "mlp": {...} | null}

    mixer of "attention":  heads, kv_heads, dim, vdim, scale, conv (taps; absent: no convolution),
                           rot {base, dims, scaling {factor, low, high, original} (absent: none)} (absent: no rotation)
    mixer of "gla":        heads, dim, vdim, tau
    mixer of "parallel":   left  {heads, kv_heads, dim, vdim, scale, rot {...}}
                           right {heads, vdim, state, groups, conv (taps), norm_groups}
                           left_scale, right_scale (absent: 1)
    mlp "dense":           ff

Every size and constant above is read here and nowhere else; the parts get them as parameters from the
plan (architectures/lufozen.py).
"""
from __future__ import annotations

from dataclasses import dataclass

from .base import ConfigError, KeyReader


@dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int
    scaling: tuple | None            # None | (factor, original, low, high)

    def to_raw(self) -> dict:
        out = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            factor, original, low, high = self.scaling
            out["scaling"] = {"factor": factor, "high": high, "low": low, "original": original}
        return out


@dataclass(frozen=True)
class AttentionConfig:
    """One softmax attention: the lone mixer (with a convolution, or none: `conv` None), or the left one of a pair."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotationConfig | None
    conv: int | None = None

    def to_raw(self) -> dict:
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.rot is not None:
            out["rot"] = self.rot.to_raw()
        if self.conv is not None:
            out["conv"] = self.conv
        return out


@dataclass(frozen=True)
class GatedLinearAttentionConfig:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int = 16                   # inner size of the decay's two matrices: a checkpoint's tensor shapes give it;
                                     # this number serves only where there is no checkpoint (random weights)

    def to_raw(self) -> dict:
        return {"dim": self.dim, "heads": self.heads, "tau": self.tau, "vdim": self.vdim}


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    def to_raw(self) -> dict:
        return {"conv": self.conv, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups,
                "state": self.state, "vdim": self.vdim}


@dataclass(frozen=True)
class PairConfig:
    left: AttentionConfig
    right: StateSpaceConfig
    left_scale: float
    right_scale: float

    def to_raw(self) -> dict:
        return {"left": self.left.to_raw(), "left_scale": self.left_scale, "right": self.right.to_raw(),
                "right_scale": self.right_scale}


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    def to_raw(self) -> dict:
        return {"ff": self.ff, "kind": "dense"}


@dataclass(frozen=True)
class LufozenLayerConfig:
    type: str                        # "parallel" | "gla" | "attention"
    mixer: object                    # PairConfig | GatedLinearAttentionConfig | AttentionConfig
    mlp: object                      # DenseConfig | None

    def to_raw(self) -> dict:
        return {"mixer": self.mixer.to_raw(), "mlp": None if self.mlp is None else self.mlp.to_raw(), "type": self.type}


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int

    def to_raw(self) -> dict:
        return {"start": self.start, "stop": self.stop, "times": self.times}


MIXER_TYPES = ("parallel", "gla", "attention")


def _sub(raw: dict, key: str, where: str) -> dict:
    v = raw.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object, got {v!r}")
    return v


def _rotation(raw: dict, dim: int):
    rot = KeyReader(raw).mapping("rot")
    if rot is None:
        return None
    r = KeyReader(rot)
    dims = r.integer("dims", minimum=0)
    if dims % 2 or dims > dim:
        raise ConfigError(f"rot.dims {dims} must be even and at most dim {dim}")
    if dims == 0:
        return None
    scaling = r.mapping("scaling")
    if scaling is not None:
        s = KeyReader(scaling)
        scaling = (s.number("factor"), s.number("original"), s.number("low"), s.number("high"))
        if scaling[2] == scaling[3]:
            raise ConfigError("rot.scaling: low and high must differ")
    return RotationConfig(r.number("base"), dims, scaling)


def _attention(raw: dict, convolved: bool) -> AttentionConfig:
    r = KeyReader(raw)
    heads, kv_heads, dim = r.integer("heads"), r.integer("kv_heads"), r.integer("dim")
    if heads % kv_heads:
        raise ConfigError(f"heads {heads} is not a multiple of kv_heads {kv_heads}")
    conv = r.integer("conv", default=None) if convolved else None
    return AttentionConfig(heads, kv_heads, dim, r.integer("vdim"), r.number("scale"), _rotation(raw, dim), conv)


def _state_space(raw: dict) -> StateSpaceConfig:
    r = KeyReader(raw)
    heads, vdim, groups, parts = r.integer("heads"), r.integer("vdim"), r.integer("groups"), r.integer("norm_groups")
    if heads % groups:
        raise ConfigError(f"right.heads {heads} is not a multiple of right.groups {groups}")
    if (heads * vdim) % parts:
        raise ConfigError(f"right.norm_groups {parts} do not divide heads * vdim = {heads * vdim}")
    return StateSpaceConfig(heads, vdim, r.integer("state"), groups, r.integer("conv"), parts)


def _mixer(kind: str, raw: dict, i: int):
    where = f"layers[{i}].mixer"
    r = KeyReader(raw)
    try:
        if kind == "attention":
            return _attention(raw, True)
        if kind == "gla":
            return GatedLinearAttentionConfig(r.integer("heads"), r.integer("dim"), r.integer("vdim"), r.number("tau"))
        if kind == "parallel":
            return PairConfig(_attention(_sub(raw, "left", where), False), _state_space(_sub(raw, "right", where)),
                              r.number("left_scale", default=1.0, positive=False),
                              r.number("right_scale", default=1.0, positive=False))
    except ConfigError as e:
        raise ConfigError(f"{e} (in {where})") from None
    raise ConfigError(f"config.json: layers[{i}].type {kind!r} is not a mixer of this architecture {MIXER_TYPES}")


def _mlp(raw, i: int):
    if raw is None:
        return None
    where = f"layers[{i}].mlp"
    if not isinstance(raw, dict):
        raise ConfigError(f"config.json: {where} must be an object or null, got {raw!r}")
    if raw.get("kind") != "dense":
        raise ConfigError(f"config.json: {where}.kind {raw.get('kind')!r} is not supported ('dense')")
    try:
        return DenseConfig(KeyReader(raw).integer("ff"))
    except ConfigError as e:
        raise ConfigError(f"{e} (in {where})") from None


@dataclass(frozen=True)
class LufozenConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    bigram_buckets: int | None       # None: no second table
    bigram_mul_prev: int
    bigram_mul_cur: int
    logit_scale: float
    loop: LoopConfig | None
    layers: tuple

    @classmethod
    def from_hf(cls, raw: dict) -> "LufozenConfig":
        r = KeyReader(raw)
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        layers = []
        for i, lr in enumerate(layers_raw):
            if not isinstance(lr, dict) or not isinstance(lr.get("type"), str):
                raise ConfigError(f"config.json: layers[{i}] must be an object with a 'type'")
            layers.append(LufozenLayerConfig(lr["type"], _mixer(lr["type"], _sub(lr, "mixer", f"layers[{i}]"), i),
                                             _mlp(lr.get("mlp"), i)))
        loop = r.mapping("loop")
        if loop is not None:
            lp = KeyReader(loop)
            loop = LoopConfig(lp.integer("start", minimum=0), lp.integer("stop"), lp.integer("times"))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"config.json: loop runs layers {loop.start} .. {loop.stop - 1} of {len(layers)}")
        norm = KeyReader(_sub(raw, "norm", "config"))
        emb = r.mapping("embedding") or {}
        bigram = KeyReader(emb).mapping("bigram")
        buckets, mul_prev, mul_cur = None, 0, 0
        if bigram is not None:
            b = KeyReader(bigram)
            buckets, mul_prev, mul_cur = b.integer("buckets"), b.integer("mul_prev", minimum=0), b.integer("mul_cur", minimum=0)
        return cls(vocab=r.integer("vocab"), width=r.integer("width"), norm_eps=norm.number("eps"),
                   embedding_scale=KeyReader(emb).number("scale", default=1.0, positive=False), bigram_buckets=buckets,
                   bigram_mul_prev=mul_prev, bigram_mul_cur=mul_cur,
                   logit_scale=r.number("logit_scale", default=1.0, positive=False), loop=loop, layers=tuple(layers))

    def running_order(self) -> list:
        """[(layer, pass)] in the order they run; `pass` is the number of the pass that starts with this run, else None."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        start, stop = self.loop.start, self.loop.stop
        order = [(i, None) for i in range(start)]
        for t in range(self.loop.times):
            order += [(i, t if i == start else None) for i in range(start, stop)]
        return order + [(i, None) for i in range(stop, n)]

    def summary(self) -> str:
        """One line for a load message."""
        kinds = [layer.type for layer in self.layers]
        loop = "" if self.loop is None else f"; layers {self.loop.start}..{self.loop.stop - 1} {self.loop.times} times"
        return (f"Lufozen: {len(kinds)}L width={self.width} ({kinds.count('attention')} convolved attention, "
                f"{kinds.count('parallel')} attention beside a state-space recurrence, {kinds.count('gla')} gated linear "
                f"attention{loop})")

    def to_hf(self) -> dict:
        """The config.json that reads back as this configuration."""
        emb = {"scale": self.embedding_scale}
        if self.bigram_buckets is not None:
            emb["bigram"] = {"buckets": self.bigram_buckets, "mul_cur": self.bigram_mul_cur,
                             "mul_prev": self.bigram_mul_prev}
        out = {"architecture": "Lufozen", "embedding": emb, "layers": [layer.to_raw() for layer in self.layers],
               "logit_scale": self.logit_scale, "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            out["loop"] = self.loop.to_raw()
        return out
