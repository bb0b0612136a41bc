"""Lufozen as a plan of parts: a decoder of pre-norm layers, some of them run several times over, whose mixers are
attention behind a short convolution, gated linear attention, or attention beside a state-space recurrence.

Embedding: `embed[token] * scale` plus a row of the hashed token-pair table `bigram`, then the norm `embed.norm`.
Layer i (tensors `l<i>.*`):  x <- x + mixer(norm1(x));  x <- x + ff(norm2(x))   (no second half without an `mlp`);
every norm is an RMS norm with a weight stored around zero (1 + w).  Layers start .. stop - 1 of `loop` run `times`
times in a row, each pass with caches and states of its own; before pass t the vector `loop.step`[t] is added to x.
mixer "attention" -> part "normed_attention": `mix.{q,k,v,o}` with `.b` biases, `mix.{q,k,v}.conv` taps, `mix.{q,k}.norm`,
rotary pairs (2i, 2i + 1) with frequencies scaled by bands of wavelength, one unit more in the softmax's denominator, a
sigmoid gate per channel `mix.g`.
mixer "gla" -> part "gated_linear_attention": `mix.{q,k,v,g,a1,a2,a2.b,norm,o}`.
mixer "parallel" -> part "side_by_side_sum": `mix.left.*` softmax attention with rotary pairs (i, i + dims/2) and the same
scaling, beside `mix.right.*` -> part "state_space": `{in,conv,conv.b,dt_bias,A_log,D,norm,o}`; the result is
left_scale * left + right_scale * right.
Feed-forward "dense": `mlp.{up,down}` with the square of relu between.
Then `final.norm` and `head`; the logits' factor is a gain on `final.norm`, whose result only the head reads.
"""
from __future__ import annotations

from ..config.lufozen import (AttentionConfig, GatedLinearAttentionConfig, LufozenConfig, PairConfig, StateSpaceConfig)
from ..config.registry import register_architecture
from ..parts.plan import LayerRun, LayerSpec, ModelPlan, PartSpec

DEFAULT_MAX_POSITIONS = 32768        # config.json gives no limit; the engine's max_model_len overrides this
NORM_OFFSET = 1.0                    # the model's norms multiply by one plus the stored weight


def _attention(m: AttentionConfig, width: int, eps: float, at: str, lone: bool) -> PartSpec:
    """`lone`: the mixer of its own (interleaved pairs, biases, convolution, one more in the denominator, gate), else the
    left one of a pair."""
    position = None
    if m.rot is not None:
        scaling = None if m.rot.scaling is None else ("bands", *m.rot.scaling)
        position = PartSpec("rotary", dict(rot_dim=m.rot.dims, theta=m.rot.base, scaling=scaling, exact=True))
    params = dict(hidden_size=width, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale,
                  norm_eps=eps, position=position, qk_norm="weighted", pairing="interleaved" if lone else "half")
    tensors = {s: at + s for s in ("q", "k", "v", "o")}
    tensors.update(q_norm=at + "q.norm", k_norm=at + "k.norm")
    if lone:
        params.update(biases=True, out_bias=True, taps=m.conv, sink="unit", channel_gate=True)
        tensors.update({f"{s}_bias": f"{at}{s}.b" for s in ("q", "k", "v", "o")}, gate=at + "g")
        if m.conv is not None:
            tensors.update({f"{s}_conv": f"{at}{s}.conv" for s in ("q", "k", "v")})
    return PartSpec("normed_attention", params, tensors)


def _linear_attention(m: GatedLinearAttentionConfig, width: int, eps: float, at: str, shapes) -> PartSpec:
    rank = m.rank                                        # the decay's inner size is the shape of its first matrix
    if shapes is not None and at + "a1" in shapes:
        rank = int(shapes[at + "a1"][0])
    tensors = {s: at + s for s in ("q", "k", "v", "g", "o", "norm", "a1", "a2")}
    return PartSpec("gated_linear_attention", dict(hidden_size=width, heads=m.heads, dim=m.dim, vdim=m.vdim, tau=m.tau,
                                                   rank=rank, norm_eps=eps), dict(tensors, a2_bias=at + "a2.b"))


def _state_space(m: StateSpaceConfig, width: int, eps: float, at: str) -> PartSpec:
    tensors = {s: at + s for s in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")}
    return PartSpec("state_space", dict(hidden_size=width, heads=m.heads, vdim=m.vdim, state=m.state, groups=m.groups,
                                        taps=m.conv, norm_parts=m.norm_groups, norm_eps=eps),
                    dict(tensors, conv_bias=at + "conv.b"))


def make_plan(cfg: LufozenConfig, tensor_names=None, tensor_shapes=None) -> ModelPlan:
    """`tensor_shapes` (name -> shape of the checkpoint's tensors, when there is a checkpoint) gives the sizes that
    config.json leaves to the tensors."""
    width, eps = cfg.width, cfg.norm_eps

    def norm(name, gain=1.0):
        return PartSpec("rmsnorm", dict(size=width, eps=eps, offset=NORM_OFFSET, gain=gain), {"weight": name})

    layers = []
    for i, layer in enumerate(cfg.layers):
        base, m = f"l{i}.", layer.mixer
        mx = base + "mix."
        if isinstance(m, PairConfig):
            mixer = PartSpec("side_by_side_sum",
                             dict(hidden_size=width, left=_attention(m.left, width, eps, mx + "left.", False),
                                  right=_state_space(m.right, width, eps, mx + "right."), left_scale=m.left_scale,
                                  right_scale=m.right_scale))
        elif isinstance(m, GatedLinearAttentionConfig):
            mixer = _linear_attention(m, width, eps, mx, tensor_shapes)
        elif isinstance(m, AttentionConfig):
            mixer = _attention(m, width, eps, mx, True)
        else:
            raise ValueError(f"layer {i}: unknown mixer configuration {m!r}")
        norms = {"mixer": norm(base + "norm1")}
        ff = None
        if layer.mlp is not None:
            ff = PartSpec("mlp", dict(hidden_size=width, intermediate_size=layer.mlp.ff, activation="relu_squared"),
                          {s: f"{base}mlp.{s}" for s in ("up", "down")})
            norms["feed_forward"] = norm(base + "norm2")
        layers.append(LayerSpec("prenorm", mixer, ff, norms))
    order = [LayerRun(i, vector=t) for i, t in cfg.running_order()]
    vectors = None
    if cfg.loop is not None:
        vectors = PartSpec("table", dict(count=cfg.loop.times, hidden_size=width), {"rows": "loop.step"})
    io = dict(vocab_size=cfg.vocab, hidden_size=width)
    embed = dict(io, scale=cfg.embedding_scale, norm_eps=eps, norm_offset=NORM_OFFSET)
    embed_tensors = {"weight": "embed", "norm": "embed.norm"}
    if cfg.bigram_buckets is not None:
        embedding = PartSpec("table_pairs", dict(embed, buckets=cfg.bigram_buckets, mul_prev=cfg.bigram_mul_prev,
                                                 mul_cur=cfg.bigram_mul_cur), dict(embed_tensors, pairs="bigram"))
    else:
        embedding = PartSpec("table", embed, embed_tensors)
    return ModelPlan(
        hidden_size=width, vocab_size=cfg.vocab, max_positions=DEFAULT_MAX_POSITIONS, embedding=embedding,
        layers=layers, order=order, final_norm=norm("final.norm", cfg.logit_scale),
        head=PartSpec("linear", io, {"weight": "head"}), vectors=vectors)


register_architecture("Lufozen", LufozenConfig, make_plan, model_types=("lufozen",))
