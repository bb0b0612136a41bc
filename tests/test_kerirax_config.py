"""Kerirax without a GPU: configuration keys, the plan of parts, running order, cache needs, shared products, the
random-weights folder, and the plain implementation's own properties (what the GPU tests lean on)."""
import copy
import json

import pytest
import torch

import kerirax_tiny as kt
import plain_kerirax as plain
from fastllm_py_b200.architectures.kerirax import make_plan
from fastllm_py_b200.cache.needs import FixedState, PagedKeysValues, PagedRows
from fastllm_py_b200.config import ConfigError, load_config
from fastllm_py_b200.config.kerirax import KeriraxConfig
from fastllm_py_b200.parts import BuildContext, Decoder, LayerRun, LayerSpec, ModelPlan, PartSpec
from fastllm_py_b200.weights import write_model_folder

RAW = kt.config([(kt.latent(3, 8, 4, 10, 12, 20), None),
                 (kt.pair(kt.left(6, 2, 12, 20, rot=8, factor=3.0), kt.right(28, 5, 3, 4), 0.6, -0.3), kt.moe(5, 3, 14)),
                 (kt.latent(2, 6, 2, 8, 8, 9), kt.dense(30)),
                 (kt.pair(kt.left(2, 1, 8, 8, rot=None), kt.right(16, 8, 2, 1)), kt.dense(8))], vocab=97, width=40, loop=(1, 3, 3))


def decoder(raw, page=8):
    cfg = KeriraxConfig.from_hf(raw)
    return cfg, Decoder(make_plan(cfg, None, tensor_shapes=kt.tensor_shapes(raw)),
                        BuildContext(torch.device("cpu"), torch.float32, page, 64))


def test_config_reads_back_and_names_every_tensor():
    cfg, dec = decoder(RAW)
    assert cfg.to_hf() == RAW
    assert KeriraxConfig.from_hf(json.loads(json.dumps(cfg.to_hf()))) == cfg
    assert dec.expected_tensors() == kt.tensor_shapes(RAW)
    assert set(dec.plan.tensor_names()) == set(kt.tensor_shapes(RAW))
    assert "Kerirax" in cfg.summary()
    for raw in (kt.config([(kt.latent(), None)], cap=None), kt.config([(kt.pair(kt.left(factor=None), kt.right()), kt.moe())], loop=(0, 1, 1))):
        cfg, dec = decoder(raw)
        assert cfg.to_hf() == raw and dec.expected_tensors() == kt.tensor_shapes(raw)
    bare = copy.deepcopy(RAW)                        # what may be absent, and what that means
    del bare["embedding"], bare["logit_softcap"], bare["loop"]
    del bare["layers"][1]["mixer"]["left_scale"], bare["layers"][1]["mixer"]["right_scale"]
    cfg, dec = decoder(bare)
    assert cfg.embedding_scale == 1.0 and dec.head.softcap is None and dec.entry is None and dec.vectors is None
    assert cfg.layers[1].mixer.left_scale == cfg.layers[1].mixer.right_scale == 1.0


def test_passes_have_caches_of_their_own_and_start_with_the_entry():
    cfg, dec = decoder(RAW)
    assert [r.layer for r in dec.order] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [r.vector for r in dec.order] == [None, 0, None, 1, None, 2, None, None]
    assert [r.entry for r in dec.order] == [r.vector is not None for r in dec.order]
    assert cfg.running_order() == plain.running_order(RAW)
    needs = dec.cache_needs()
    assert needs[0] == PagedRows(16, None)
    for run in (1, 3, 5):
        assert needs[(run, "left")] == PagedKeysValues(2, 12, 20, None)
        assert needs[(run, "right")] == FixedState((28 * 5 + 3 * 28,), "float32")
    for run in (2, 4, 6):
        assert needs[run] == PagedRows(10, None)
    assert needs[(7, "right")] == FixedState((16 * 8,), "float32")                     # one tap keeps no inputs


def test_layers_share_a_norm_and_the_pair_holds_two_products():
    _, dec = decoder(RAW)
    w = {k: v.float() for k, v in kt.weights(RAW, seed=1).items()}
    dec.load(w)
    block = dec.blocks[1]
    assert block.norm_ff is None and block.feed_forward is not None and block.mixer.partial_side
    sides = block.mixer
    cols = 6 * 12 + 2 * 12 + 2 * 20 + 6
    assert sides.left.in_cols == cols and sides.right_at == 144 and sides.in_cols == 144 + 56
    assert tuple(sides.proj.weight.shape) == (200, 40) and tuple(sides.o.weight.shape) == (40, 6 * 20 + 28)
    assert torch.equal(sides.proj.weight[cols - 6:cols], w["l1.mix.left.g"])
    assert float(sides.proj.weight[cols:144].abs().max()) == 0.0
    assert torch.equal(sides.proj.weight[144:], w["l1.mix.right.in"])
    assert torch.equal(sides.o.weight[:, 120:], w["l1.mix.right.o"])
    assert sides.left.result_scale == 0.6 and sides.right.result_scale == -0.3
    assert torch.allclose(sides.right.a, -torch.exp(w["l1.mix.right.A_log"]))
    assert torch.equal(dec.blocks[0].mixer.sink, w["l0.mix.sink"])
    assert torch.equal(dec.entry.linear.weight, w["loop.in"])
    ff = block.feed_forward
    assert ff.on_input and ff.activation_params == (1.5, 1.702) and not ff.choice_bias and ff.top == 3


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "conv", "type"),
    (("layers", 0, "mixer", "rot_dim"), 6, "rot_dim"),
    (("layers", 0, "mixer", "rot"), None, "rot_dim"),
    (("layers", 0, "mixer", "q_rank"), None, "q_rank"),
    (("layers", 1, "mixer", "left", "kv_heads"), 4, "kv_heads"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 7, "rot.dims"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 14, "rot.dims"),
    (("layers", 1, "mixer", "left", "rot", "scaling", "factor"), "big", "factor"),
    (("layers", 1, "mixer", "right", "dt_rank"), 0, "dt_rank"),
    (("layers", 1, "mixer", "right", "conv"), 0, "conv"),
    (("layers", 1, "mixer", "right"), None, "right"),
    (("layers", 1, "mixer", "left_scale"), "much", "left_scale"),
    (("layers", 1, "mlp", "router", "top"), 6, "top"),
    (("layers", 1, "mlp", "expert", "limit"), 0, "limit"),
    (("layers", 1, "mlp", "kind"), "sparse", "kind"),
    (("layers", 2, "mlp", "ff"), None, "ff"),
    (("loop", "stop"), 5, "loop"),
    (("loop", "start"), 3, "loop"),
    (("logit_softcap",), -1.0, "logit_softcap"),
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
        KeriraxConfig.from_hf(raw)


def test_a_written_folder_loads_by_its_architecture_string(tmp_path):
    cfg = KeriraxConfig.from_hf(RAW)
    folder = write_model_folder(cfg, tmp_path / "m", seed=3)
    arch, again = load_config(folder)
    assert arch.name == "Kerirax" and again == cfg
    from safetensors import safe_open

    with safe_open(str(folder / "model.safetensors"), framework="pt") as f:
        assert {k: tuple(f.get_slice(k).get_shape()) for k in f.keys()} == kt.tensor_shapes(RAW)


def test_a_run_cannot_start_with_an_entry_the_plan_lacks():
    io = dict(vocab_size=8, hidden_size=8)
    norm = PartSpec("rmsnorm", dict(size=8, eps=1e-5), {"weight": "n"})
    mixer = PartSpec("gated_linear_attention", dict(hidden_size=8, heads=1, dim=4, vdim=4, tau=1.0, rank=2, norm_eps=1e-5), {})
    plan = ModelPlan(hidden_size=8, vocab_size=8, max_positions=16, embedding=PartSpec("table", io, {"weight": "e"}),
                     layers=[LayerSpec("prenorm", mixer, None, {"mixer": norm})], order=[LayerRun(0, entry=True)],
                     final_norm=norm, head=PartSpec("linear", io, {"weight": "h"}))
    with pytest.raises(ValueError, match="entry"):
        plan.validate()


def test_rotary_tables_follow_the_linear_scaling():
    from fastllm_py_b200.parts import build_part

    for factor in (None, 4.0, 2.5):
        spec = PartSpec("rotary", dict(rot_dim=12, theta=50000.0, scaling=None if factor is None else ("linear", factor), exact=True))
        cos, sin = build_part("position", spec, BuildContext(torch.device("cpu"), torch.float32, 8, 300)).tables()
        f = plain.rotary_frequencies(12, 50000.0, None if factor is None else {"factor": factor})
        ang = torch.arange(300, dtype=torch.float64)[:, None] * f[None, :]
        assert torch.allclose(cos.double(), torch.cos(ang), atol=1e-6) and torch.allclose(sin.double(), torch.sin(ang), atol=1e-6)


ALTERS = ("no_rejoin", "swapped_rejoin", "no_step", "no_query_norm", "no_sink", "head_norm", "no_scaling", "other_pairing", "no_gate",
          "no_dt_bias", "no_skip", "swapped_scales", "renormalised", "weight_on_output", "one_after_the_other", "no_cap")


def test_plain_implementation_is_causal_and_every_mechanism_matters():
    raw = kt.config([(kt.pair(kt.left(4, 2, 8, 8, rot=8, scale=1.0), kt.right(20, 6, 4, 3), 0.9, 0.5), kt.dense(16)),
                     (kt.latent(2, 8, 4, 6, 8, 12, scale=1.0), kt.moe(5, 2, 12))], width=24, vocab=30, loop=(0, 2, 2), cap=4.0)
    w = kt.weights(raw, seed=1, slow=True)
    toks = list(range(3, 26))
    full = plain.forward(raw, w, toks)
    assert torch.allclose(plain.forward(raw, w, toks[:11]), full[:11], atol=1e-12)
    for alter in ALTERS:
        assert float((plain.forward(raw, w, toks, alter={alter}) - full).abs().max()) > 1e-3, alter
    # a state handed on equals the whole sequence
    h = torch.randn(17, 24, dtype=torch.float64, generator=torch.Generator().manual_seed(2))
    t, m = plain.sub(w, "l0.mix.right."), raw["layers"][0]["mixer"]["right"]
    whole, _ = plain.selective_scan(h, t, m)
    head, state = plain.selective_scan(h[:6], t, m)
    rest, _ = plain.selective_scan(h[6:], t, m, state)
    assert torch.allclose(torch.cat([head, rest]), whole, atol=1e-12)
