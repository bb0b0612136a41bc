"""KeriraxConfig: the typed configuration of the Kerirax decoder.

A Kerirax model is a list of parallel layers (one norm, whose result both the mixer and the feed-forward read), some of
which run several times in a row with the same weights, each such pass starting with a product of the stream beside the
embedding output.  Its config.json is nested:

    architecture     "Kerirax"
    vocab, width     sizes of the embedding table and the residual stream
    norm.eps         the epsilon of every norm
    embedding        {"scale": s}   (absent: 1)
    loop             {"start", "stop", "times"}: layers start .. stop - 1 run `times` times in a row (absent: every layer
                     runs once)
    logit_softcap    the logits' soft cap (absent: none)
    layers[i]        {"type": "parallel" | "latent_attention", "mixer": {...}, "mlp": {...} | null}

    mixer of "latent_attention":  heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, rot {base, dims = rot_dim}
    mixer of "parallel":   left  {heads, kv_heads, dim, vdim, scale,
                                  rot {base, dims, scaling {factor} (absent: none)} (absent: no rotation)}
                           right {inner, state, dt_rank, conv (taps)}
                           left_scale, right_scale (absent: 1)
    mlp "dense":           ff
    mlp "moe":             expert {ff, limit}, router {experts, top}

Every size and constant above is read here and nowhere else; the parts get them as parameters from the
plan (architectures/kerirax.py).
"""
from __future__ import annotations

from dataclasses import dataclass

from .base import ConfigError, KeyReader


@dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int
    factor: float | None             # of a linear scaling

    def to_raw(self) -> dict:
        out = {"base": self.base, "dims": self.dims}
        if self.factor is not None:
            out["scaling"] = {"factor": self.factor}
        return out


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: RotationConfig

    def to_raw(self) -> dict:
        return {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "q_rank": self.q_rank, "rot": self.rot.to_raw(),
                "rot_dim": self.rot_dim, "scale": self.scale, "vdim": self.vdim}


@dataclass(frozen=True)
class AttentionConfig:
    """The softmax attention of a pair."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotationConfig | None

    def to_raw(self) -> dict:
        out = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.rot is not None:
            out["rot"] = self.rot.to_raw()
        return out


@dataclass(frozen=True)
class SelectiveScanConfig:
    """The recurrence of a pair."""
    inner: int
    state: int
    dt_rank: int
    conv: int

    def to_raw(self) -> dict:
        return {"conv": self.conv, "dt_rank": self.dt_rank, "inner": self.inner, "state": self.state}


@dataclass(frozen=True)
class PairConfig:
    left: AttentionConfig
    right: SelectiveScanConfig
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
class ExpertsConfig:
    experts: int
    top: int
    ff: int
    limit: float

    def to_raw(self) -> dict:
        return {"expert": {"ff": self.ff, "limit": self.limit}, "kind": "moe",
                "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class KeriraxLayerConfig:
    type: str                        # "parallel" | "latent_attention"
    mixer: object                    # PairConfig | LatentConfig
    mlp: object                      # DenseConfig | ExpertsConfig | None

    def to_raw(self) -> dict:
        return {"mixer": self.mixer.to_raw(), "mlp": None if self.mlp is None else self.mlp.to_raw(), "type": self.type}


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int

    def to_raw(self) -> dict:
        return {"start": self.start, "stop": self.stop, "times": self.times}


MIXER_TYPES = ("parallel", "latent_attention")


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
        raise ConfigError(f"rot.dims {dims} must be even and at most {dim}")
    scaling = r.mapping("scaling")
    return RotationConfig(r.number("base"), dims, None if scaling is None else KeyReader(scaling).number("factor"))


def _attention(raw: dict) -> AttentionConfig:
    r = KeyReader(raw)
    heads, kv_heads, dim = r.integer("heads"), r.integer("kv_heads"), r.integer("dim")
    if heads % kv_heads:
        raise ConfigError(f"left.heads {heads} is not a multiple of left.kv_heads {kv_heads}")
    return AttentionConfig(heads, kv_heads, dim, r.integer("vdim"), r.number("scale"), _rotation(raw, dim))


def _latent(raw: dict) -> LatentConfig:
    r = KeyReader(raw)
    rot_dim = r.integer("rot_dim")
    rot = _rotation(raw, rot_dim)
    if rot is None or rot.dims != rot_dim:
        raise ConfigError(f"rot.dims must be rot_dim = {rot_dim}")
    return LatentConfig(r.integer("heads"), r.integer("dim"), rot_dim, r.integer("vdim"), r.integer("kv_rank"),
                        r.integer("q_rank"), r.number("scale"), rot)


def _mixer(kind: str, raw: dict, i: int):
    where = f"layers[{i}].mixer"
    r = KeyReader(raw)
    try:
        if kind == "latent_attention":
            return _latent(raw)
        if kind == "parallel":
            s = KeyReader(_sub(raw, "right", where))
            right = SelectiveScanConfig(s.integer("inner"), s.integer("state"), s.integer("dt_rank"), s.integer("conv"))
            return PairConfig(_attention(_sub(raw, "left", where)), right, r.number("left_scale", default=1.0, positive=False),
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
    kind = raw.get("kind")
    try:
        if kind == "dense":
            return DenseConfig(KeyReader(raw).integer("ff"))
        if kind == "moe":
            e, r = KeyReader(_sub(raw, "expert", where)), KeyReader(_sub(raw, "router", where))
            experts, top = r.integer("experts"), r.integer("top")
            if top > experts:
                raise ConfigError(f"router.top {top} of {experts} experts")
            return ExpertsConfig(experts, top, e.integer("ff"), e.number("limit"))
    except ConfigError as e:
        raise ConfigError(f"{e} (in {where})") from None
    raise ConfigError(f"config.json: {where}.kind {kind!r} is not supported ('dense', 'moe')")


@dataclass(frozen=True)
class KeriraxConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    logit_softcap: float | None
    loop: LoopConfig | None
    layers: tuple

    @classmethod
    def from_hf(cls, raw: dict) -> "KeriraxConfig":
        r = KeyReader(raw)
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config.json: layers must be a list with at least one layer")
        layers = []
        for i, lr in enumerate(layers_raw):
            if not isinstance(lr, dict) or not isinstance(lr.get("type"), str):
                raise ConfigError(f"config.json: layers[{i}] must be an object with a 'type'")
            layers.append(KeriraxLayerConfig(lr["type"], _mixer(lr["type"], _sub(lr, "mixer", f"layers[{i}]"), i),
                                             _mlp(lr.get("mlp"), i)))
        loop = r.mapping("loop")
        if loop is not None:
            lp = KeyReader(loop)
            loop = LoopConfig(lp.integer("start", minimum=0), lp.integer("stop"), lp.integer("times"))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"config.json: loop runs layers {loop.start} .. {loop.stop - 1} of {len(layers)}")
        norm = KeyReader(_sub(raw, "norm", "config"))
        emb = KeyReader(r.mapping("embedding") or {})
        return cls(vocab=r.integer("vocab"), width=r.integer("width"), norm_eps=norm.number("eps"),
                   embedding_scale=emb.number("scale", default=1.0, positive=False),
                   logit_softcap=None if raw.get("logit_softcap") is None else r.number("logit_softcap"), loop=loop,
                   layers=tuple(layers))

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
        moe = sum(isinstance(layer.mlp, ExpertsConfig) for layer in self.layers)
        loop = "" if self.loop is None else f"; layers {self.loop.start}..{self.loop.stop - 1} {self.loop.times} times"
        return (f"Kerirax: {len(kinds)}L width={self.width} ({kinds.count('latent_attention')} latent attention, "
                f"{kinds.count('parallel')} attention beside a selective scan; {moe} with experts{loop})")

    def to_hf(self) -> dict:
        """The config.json that reads back as this configuration."""
        out = {"architecture": "Kerirax", "embedding": {"scale": self.embedding_scale},
               "layers": [layer.to_raw() for layer in self.layers], "norm": {"eps": self.norm_eps}, "vocab": self.vocab,
               "width": self.width}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            out["loop"] = self.loop.to_raw()
        return out
