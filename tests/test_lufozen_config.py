"""Lufozen without a GPU: configuration keys, the plan of parts, running order, cache needs, shared products, the
random-weights folder, and the plain implementation's own properties (what the GPU tests lean on)."""
import copy
import json

import pytest
import torch

import lufozen_tiny as lt
import plain_lufozen as plain
from fastllm_py_b200.architectures.lufozen import make_plan
from fastllm_py_b200.cache.needs import FixedState, PagedKeysValues
from fastllm_py_b200.config import ConfigError, load_config
from fastllm_py_b200.config.lufozen import LufozenConfig
from fastllm_py_b200.parts import BuildContext, Decoder, LayerRun, LayerSpec, ModelPlan, PartSpec
from fastllm_py_b200.weights import write_model_folder

BANDS = (8.0, 64, 1.0, 4.0)
RAW = lt.config([(lt.linear(3, 8, 12, 8.0), None),
                 (lt.attention(6, 2, 12, 20, conv=3, rot=8, scaling=BANDS), lt.dense(48)),
                 (lt.pair(lt.left(4, 2, 16, 24, rot=16), lt.right(6, 4, 10, 3, conv=4, norm_groups=2), 0.6, 0.3), lt.dense(30)),
                 (lt.attention(2, 1, 8, 8, conv=1, rot=None), None),
                 (lt.linear(1, 4, 4, 1.0), lt.dense(8))], vocab=97, width=40, loop=(1, 3, 3))


def decoder(raw, page=8, rank=6):
    cfg = LufozenConfig.from_hf(raw)
    plan = make_plan(cfg, None, tensor_shapes=lt.tensor_shapes(raw, rank))
    return cfg, Decoder(plan, BuildContext(torch.device("cpu"), torch.float32, page, 64))


def test_config_reads_back_and_names_every_tensor():
    cfg, dec = decoder(RAW)
    assert cfg.to_hf() == RAW
    assert LufozenConfig.from_hf(json.loads(json.dumps(cfg.to_hf()))) == cfg
    assert dec.expected_tensors() == lt.tensor_shapes(RAW)
    assert set(dec.plan.tensor_names()) == set(lt.tensor_shapes(RAW))
    assert "Lufozen" in cfg.summary()
    _, other = decoder(RAW, rank=11)                 # the decay's inner size comes from the checkpoint's shapes
    assert other.expected_tensors()["l0.mix.a1"] == (11, 40)
    for raw in (lt.config([(lt.linear(), None)], buckets=None), lt.config([(lt.attention(conv=None), lt.dense())])):
        cfg, dec = decoder(raw)
        assert cfg.to_hf() == raw and dec.expected_tensors() == lt.tensor_shapes(raw)


def test_loop_runs_layers_again_with_caches_of_their_own():
    cfg, dec = decoder(RAW)
    assert len(dec.blocks) == 5 and [r.layer for r in dec.order] == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert [r.vector for r in dec.order] == [None, 0, None, 1, None, 2, None, None, None]
    assert [(i, t) for i, t in cfg.running_order()] == plain.running_order(RAW)
    needs = dec.cache_needs()
    assert needs[0] == FixedState((3 * 12 * 8,), "float32")
    for run in (1, 3, 5):                            # keys and values, and two projected rows of q | k | v
        assert needs[(run, "kv")] == PagedKeysValues(2, 12, 20, None)
        assert needs[(run, "conv")] == FixedState((2 * (6 * 12 + 2 * 12 + 2 * 20),), "float32")
    for run in (2, 4, 6):
        assert needs[(run, "left")] == PagedKeysValues(2, 16, 24, None)
        inner, channels = 6 * 4, 6 * 4 + 2 * 3 * 10
        assert needs[(run, "right")] == FixedState((-(-(inner * 10 + 3 * channels) // 4) * 4,), "float32")
    assert needs[7] == PagedKeysValues(1, 8, 8, None)              # one tap keeps no rows
    assert needs["embedding"] == FixedState((1,), "int32")
    whole = copy.deepcopy(RAW)
    whole["loop"] = {"start": 0, "stop": 5, "times": 1}
    assert [r.vector for r in decoder(whole)[1].order] == [0, None, None, None, None]


def test_the_pair_holds_two_products_for_four():
    _, dec = decoder(RAW)
    sides = dec.blocks[2].mixer
    assert sides.in_cols == (4 + 2) * 16 + 2 * 24 + 2 * 24 + 2 * 3 * 10 + 6 and sides.out_cols == 4 * 24 + 24
    w = {k: v.float() for k, v in lt.weights(RAW, seed=1).items()}
    dec.load(w)
    assert tuple(sides.proj.weight.shape) == (sides.in_cols, 40) and tuple(sides.o.weight.shape) == (40, sides.out_cols)
    assert torch.equal(sides.o.weight[:, 4 * 24:], w["l2.mix.right.o"]) and sides.left.proj is None
    assert torch.equal(sides.proj.weight[:64], w["l2.mix.left.q"])
    assert sides.left.result_scale == 0.6
    assert torch.allclose(sides.right.norm_w, w["l2.mix.right.norm"] * 0.3)
    # norms stored around zero, the logits' factor on the last one, a bias that the block adds to the stream
    assert torch.allclose(dec.blocks[1].norm_mixer.weight, 1.0 + w["l1.norm1"])
    assert torch.allclose(dec.final_norm.weight, (1.0 + w["final.norm"]) * 0.7)
    assert torch.allclose(dec.embedding.norm_w, 1.0 + w["embed.norm"])
    assert dec.blocks[1].mixer.defers_out_bias and torch.equal(dec.blocks[1].mixer.out_bias, w["l1.mix.o.b"])
    assert torch.equal(dec.vectors.row(2), w["loop.step"][2])


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "conv", "type"),
    (("layers", 0, "mixer", "tau"), 0, "tau"),
    (("layers", 1, "mixer", "kv_heads"), 4, "kv_heads"),
    (("layers", 1, "mixer", "rot", "dims"), 7, "rot.dims"),
    (("layers", 1, "mixer", "rot", "dims"), 14, "rot.dims"),
    (("layers", 1, "mixer", "rot", "scaling", "factor"), "big", "factor"),
    (("layers", 1, "mixer", "rot", "scaling", "high"), 1.0, "low and high"),
    (("layers", 1, "mixer", "conv"), 0, "conv"),
    (("layers", 1, "mlp", "kind"), "moe", "kind"),
    (("layers", 1, "mlp", "ff"), None, "ff"),
    (("layers", 2, "mixer", "right", "groups"), 4, "groups"),
    (("layers", 2, "mixer", "right", "norm_groups"), 5, "norm_groups"),
    (("layers", 2, "mixer", "right"), None, "right"),
    (("layers", 2, "mixer", "left_scale"), "much", "left_scale"),
    (("loop", "stop"), 6, "loop"),
    (("loop", "start"), 3, "loop"),
    (("embedding", "bigram", "buckets"), 0, "buckets"),
    (("norm", "eps"), 0, "eps"),
    (("width",), "wide", "width"),
])
def test_wrong_values_are_refused_by_name(path, value, word):
    raw = copy.deepcopy(RAW)
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        LufozenConfig.from_hf(raw)


def test_a_written_folder_loads_by_its_architecture_string(tmp_path):
    cfg = LufozenConfig.from_hf(RAW)
    folder = write_model_folder(cfg, tmp_path / "m", seed=3)
    arch, again = load_config(folder)
    assert arch.name == "Lufozen" and again == cfg
    from safetensors import safe_open

    with safe_open(str(folder / "model.safetensors"), framework="pt") as f:
        assert {k: tuple(f.get_slice(k).get_shape()) for k in f.keys()} == lt.tensor_shapes(RAW, rank=16)


def test_a_run_cannot_start_with_a_vector_the_plan_lacks():
    io = dict(vocab_size=8, hidden_size=8)
    norm = PartSpec("rmsnorm", dict(size=8, eps=1e-5), {"weight": "n"})
    mixer = PartSpec("gated_linear_attention", dict(hidden_size=8, heads=1, dim=4, vdim=4, tau=1.0, rank=2, norm_eps=1e-5), {})
    plan = ModelPlan(hidden_size=8, vocab_size=8, max_positions=16, embedding=PartSpec("table", io, {"weight": "e"}),
                     layers=[LayerSpec("prenorm", mixer, None, {"mixer": norm})], order=[LayerRun(0, vector=0)],
                     final_norm=norm, head=PartSpec("linear", io, {"weight": "h"}))
    with pytest.raises(ValueError, match="vector"):
        plan.validate()


def test_rotary_tables_follow_the_bands():
    from fastllm_py_b200.parts import build_part

    for scaling in (None, BANDS, (4.0, 512, 1.0, 4.0)):
        spec = PartSpec("rotary", dict(rot_dim=12, theta=250000.0, scaling=None if scaling is None else ("bands", *scaling), exact=True))
        cos, sin = build_part("position", spec, BuildContext(torch.device("cpu"), torch.float32, 8, 300)).tables()
        raw = None if scaling is None else dict(zip(("factor", "original", "low", "high"), scaling))
        ang = torch.arange(300, dtype=torch.float64)[:, None] * plain.rotary_frequencies(12, 250000.0, raw)[None, :]
        assert torch.allclose(cos.double(), torch.cos(ang), atol=1e-6) and torch.allclose(sin.double(), torch.sin(ang), atol=1e-6)


def test_plain_implementation_is_causal_and_every_mechanism_matters():
    raw = lt.config([(lt.attention(4, 2, 8, 8, conv=3, rot=8, scale=1.0), lt.dense(16)),
                     (lt.pair(lt.left(2, 1, 8, 8, rot=8, scale=1.0), lt.right(4, 6, 5, 2, 3, 4), 0.8, 0.3), None),
                     (lt.linear(2, 4, 6, 4.0), None)], width=24, vocab=30, loop=(0, 2, 2))
    w = lt.weights(raw, seed=1, slow=True)
    toks = list(range(3, 26))
    full = plain.forward(raw, w, toks)
    assert torch.allclose(plain.forward(raw, w, toks[:11]), full[:11], atol=1e-12)
    for alter in ("no_conv", "other_pairing", "no_sink", "left_sink", "no_gate", "no_out_bias", "no_skip", "one_norm", "norm_first",
                  "no_decay", "swapped_scales", "no_step", "no_pairs", "plain_weight"):
        assert float((plain.forward(raw, w, toks, alter={alter}) - full).abs().max()) > 1e-3, alter
    moved = plain.forward(raw, w, [toks[0] + 1] + toks[1:])
    assert float((moved - full)[-1].abs().max()) > 1e-6                                 # the states reach back
    # states handed on equal whole sequences
    h = torch.randn(17, 24, dtype=torch.float64, generator=torch.Generator().manual_seed(2))
    t, m = plain.sub(w, "l1.mix.right."), raw["layers"][1]["mixer"]["right"]
    whole, _ = plain.state_space(h, t, m, 1e-5)
    head, state = plain.state_space(h[:6], t, m, 1e-5)
    rest, _ = plain.state_space(h[6:], t, m, 1e-5, state)
    assert torch.allclose(torch.cat([head, rest]), whole, atol=1e-12)
    t, m = plain.sub(w, "l2.mix."), raw["layers"][2]["mixer"]
    whole, _ = plain.gated_linear_attention(h, t, m, 1e-5)
    head, state = plain.gated_linear_attention(h[:9], t, m, 1e-5)
    rest, _ = plain.gated_linear_attention(h[9:], t, m, 1e-5, state)
    assert torch.allclose(torch.cat([head, rest]), whole, atol=1e-12)
