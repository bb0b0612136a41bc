"""Kerirax as a plan of parts: a decoder of parallel layers behind one norm each, some of them run several times over, whose
mixers are latent attention with a sink or attention beside a selective scan.

Embedding: `embed[token] * scale`.
Layer i (tensors `l<i>.*`):  h = norm1(x);  x <- x + (mixer(h) + ff(h))   (mixer alone without an `mlp`).
Layers start .. stop - 1 of `loop` run `times` times in a row, each pass with caches and states of its own; before pass t
x <- `loop.in` [x; embedding output], then the vector `loop.step`[t] is added to x.
mixer "latent_attention" -> part "latent_attention": `mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,o,sink}`, queries through a
latent, rotary pairs (2i, 2i + 1).
mixer "parallel" -> part "side_by_side_sum": `mix.left.{q,k,v,o,g}` softmax attention with norms over the whole query and key
projections (`q.norm`, `k.norm`), rotary pairs (2i, 2i + 1) and a sigmoid gate per head, beside `mix.right.*` -> part
"selective_scan": `{in,conv,conv.b,x,dt,dt.b,A_log,D,o}`; the result is left_scale * left + right_scale * right.
Feed-forward "dense": `mlp.{gate,up,down}` with silu; "moe": `mlp.router` and `mlp.e<j>.{gate,up,down}`, clamped swish units
chosen by sigmoid score, the score multiplying what the expert reads.
Then `final.norm`, `head` and the logits' soft cap.
"""
from __future__ import annotations

from ..config.kerirax import AttentionConfig, ExpertsConfig, KeriraxConfig, LatentConfig, PairConfig, SelectiveScanConfig
from ..config.registry import register_architecture
from ..parts.plan import LayerRun, LayerSpec, ModelPlan, PartSpec

DEFAULT_MAX_POSITIONS = 32768        # config.json gives no limit; the engine's max_model_len overrides this
SWISH_SLOPE = 1.702                  # of the experts' units


def _rotary(rot) -> PartSpec:
    scaling = None if rot.factor is None else ("linear", rot.factor)
    return PartSpec("rotary", dict(rot_dim=rot.dims, theta=rot.base, scaling=scaling, exact=True))


def _attention(m: AttentionConfig, width: int, eps: float, at: str) -> PartSpec:
    position = _rotary(m.rot) if m.rot is not None and m.rot.dims else None
    tensors = {s: at + s for s in ("q", "k", "v", "o")}
    return PartSpec("normed_attention",
                    dict(hidden_size=width, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale,
                         norm_eps=eps, position=position, qk_norm="whole", pairing="interleaved", head_gate=True),
                    dict(tensors, q_norm=at + "q.norm", k_norm=at + "k.norm", gate=at + "g"))


def _selective_scan(m: SelectiveScanConfig, width: int, at: str) -> PartSpec:
    tensors = {s: at + s for s in ("in", "conv", "x", "dt", "A_log", "D", "o")}
    return PartSpec("selective_scan", dict(hidden_size=width, inner=m.inner, state=m.state, rank=m.dt_rank, taps=m.conv),
                    dict(tensors, conv_bias=at + "conv.b", dt_bias=at + "dt.b"))


def _latent(m: LatentConfig, width: int, eps: float, at: str) -> PartSpec:
    tensors = {s: at + s for s in ("dq", "uq", "dkv", "uk", "uv", "o", "sink")}
    return PartSpec("latent_attention",
                    dict(hidden_size=width, heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, kv_rank=m.kv_rank,
                         q_rank=m.q_rank, scale=m.scale, window=None, norm_eps=eps, position=_rotary(m.rot),
                         pairing="interleaved", sink=True),
                    dict(tensors, dq_norm=at + "dq.norm", dkv_norm=at + "dkv.norm"))


def _feed_forward(m, width: int, at: str):
    if m is None:
        return None
    if not isinstance(m, ExpertsConfig):
        return PartSpec("swiglu", dict(hidden_size=width, intermediate_size=m.ff), {s: at + s for s in ("gate", "up", "down")})
    tensors = {"router": at + "router"}
    for e in range(m.experts):
        tensors.update({f"{s}.{e}": f"{at}e{e}.{s}" for s in ("gate", "up", "down")})
    return PartSpec("routed_experts", dict(hidden_size=width, experts=m.experts, top=m.top, expert_ff=m.ff, score="sigmoid",
                                           activation="clamped_swish", activation_params=(m.limit, SWISH_SLOPE),
                                           weight_on="input", choice_bias=False), tensors)


def make_plan(cfg: KeriraxConfig, tensor_names=None, tensor_shapes=None) -> ModelPlan:
    width, eps = cfg.width, cfg.norm_eps

    def norm(name):
        return PartSpec("rmsnorm", dict(size=width, eps=eps), {"weight": name})

    layers = []
    for i, layer in enumerate(cfg.layers):
        base, m = f"l{i}.", layer.mixer
        mx = base + "mix."
        if isinstance(m, PairConfig):
            mixer = PartSpec("side_by_side_sum",
                             dict(hidden_size=width, left=_attention(m.left, width, eps, mx + "left."),
                                  right=_selective_scan(m.right, width, mx + "right."), left_scale=m.left_scale,
                                  right_scale=m.right_scale))
        elif isinstance(m, LatentConfig):
            mixer = _latent(m, width, eps, mx)
        else:
            raise ValueError(f"layer {i}: unknown mixer configuration {m!r}")
        layers.append(LayerSpec("parallel", mixer, _feed_forward(layer.mlp, width, base + "mlp."), {"mixer": norm(base + "norm1")}))
    vectors = entry = None
    if cfg.loop is not None:
        vectors = PartSpec("table", dict(count=cfg.loop.times, hidden_size=width), {"rows": "loop.step"})
        entry = PartSpec("rejoin", dict(hidden_size=width), {"weight": "loop.in"})
    io = dict(vocab_size=cfg.vocab, hidden_size=width)
    return ModelPlan(
        hidden_size=width, vocab_size=cfg.vocab, max_positions=DEFAULT_MAX_POSITIONS,
        embedding=PartSpec("table", dict(io, scale=cfg.embedding_scale), {"weight": "embed"}), layers=layers,
        order=[LayerRun(i, vector=t, entry=t is not None) for i, t in cfg.running_order()], final_norm=norm("final.norm"),
        head=PartSpec("linear", dict(io, softcap=cfg.logit_softcap), {"weight": "head"}), vectors=vectors, entry=entry)


register_architecture("Kerirax", KeriraxConfig, make_plan, model_types=("kerirax",))
