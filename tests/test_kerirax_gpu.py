"""Kerirax in the engine against the plain implementation (tests/plain_kerirax.py).

Small configurations with weights of their own (tests/kerirax_tiny.py).  The 32-bit engine is
held to 2e-4 of the largest logit against the float64 oracle and, cut against cut, to bitwise
equality (every kernel of that path sums in an order that depends on the token's own place
only); the bfloat16 engine's error, position by position, to a fraction of the logits' spread.
Every engine runs with the cache's check mode on (pages that go back are overwritten) and with
fewer state slots than requests, so pages and slots are used again.
"""
import numpy as np
import pytest
import torch

import kerirax_tiny as kt
import plain_kerirax as plain
import replay
from test_kerirax_config import ALTERS

pytestmark = pytest.mark.gpu

# every size differs from model to model, and some are the degenerate values: one head, heads == kv_heads, groups of three
# and twelve query heads, one tap, nine taps, no rotation, part of the dimensions rotated, one expert, all experts chosen, a
# state of one, a rank of one, no loop, a loop over all layers, over one layer, run once, layers without feed-forward in
# every place, no soft cap, widths that are multiples of neither 8 nor 32
MODELS = {
    "mix": dict(layers=[(kt.pair(kt.left(4, 2, 16, 12, rot=8, factor=4.0), kt.right(36, 12, 5, 4), 0.8, 0.6), kt.dense(48)),
                        (kt.latent(3, 12, 8, 20, 16, 24), kt.moe(6, 2, 24)),
                        (kt.pair(kt.left(6, 2, 12, 20, rot=12, factor=None), kt.right(28, 7, 3, 3)), kt.moe(4, 1, 20)),
                        (kt.latent(2, 8, 4, 8, 12, 10), None)],
                kw=dict(vocab=97, width=40, loop=(1, 3, 2)), page=8),
    "odd": dict(layers=[(kt.latent(1, 7, 2, 5, 9, 11, base=300.0), kt.moe(1, 1, 9)),
                        (kt.pair(kt.left(12, 1, 6, 5, rot=None), kt.right(13, 1, 1, 9), -0.5, 1.3), None),
                        (kt.pair(kt.left(3, 3, 10, 7, rot=6, base=500.0, factor=3.0), kt.right(21, 33, 9, 1), 1.0, 1.0), kt.moe(3, 3, 7)),
                        (kt.latent(5, 10, 6, 9, 20, 6), kt.dense(11))],
                kw=dict(vocab=61, width=36, eps=1e-6, loop=(0, 4, 2), scale=1.0, cap=None), page=16),
    # sizes that the tensor-core kernels take in bfloat16 (multiples of 16 or 32 throughout)
    "even": dict(layers=[(kt.pair(kt.left(8, 2, 32, 64, rot=32, factor=8.0), kt.right(96, 16, 16, 4), 0.5, 0.8), kt.dense(128)),
                         (kt.latent(4, 32, 16, 32, 32, 64), kt.moe(8, 2, 64, 3.0)),
                         (kt.pair(kt.left(4, 4, 64, 32, rot=16, factor=2.0), kt.right(64, 64, 8, 2), 1.1, 0.9), kt.moe(4, 2, 32))],
                 kw=dict(vocab=80, width=64, loop=(2, 3, 1)), page=16),
    "single": dict(layers=[(kt.pair(kt.left(2, 1, 16, 16, rot=16), kt.right(48, 130, 8, 4)), kt.dense(32))],
                   kw=dict(vocab=50, width=48), page=4),
}
LENGTHS = {"mix": [1, 2, 9, 23, 40, 77], "odd": [3, 30, 64, 51], "even": [150, 70, 90], "single": [33, 5, 61]}


@pytest.fixture(scope="module")
def made(tmp_path_factory):
    root = tmp_path_factory.mktemp("kerirax")
    out = {}
    for k, (name, m) in enumerate(MODELS.items()):
        raw = kt.config(m["layers"], **m["kw"])
        w = kt.weights(raw, seed=5 + k)
        rng = np.random.default_rng(40 + k)
        requests = {f"q{i}": rng.integers(0, raw["vocab"], size=n).tolist() for i, n in enumerate(LENGTHS[name])}
        want = {rid: plain.forward(raw, w, toks).float() for rid, toks in requests.items()}
        out[name] = dict(raw=raw, weights=w, folder=kt.write(raw, w, root / name), requests=requests, want=want,
                         page=m["page"])
    return out


_engines = {}


def engine(made, name, dtype, max_tokens=None, max_requests=3, graph=False):
    from fastllm_py_b200 import Model

    key = (name, dtype, max_tokens, max_requests, graph)
    if key not in _engines:
        _engines[key] = Model.load(made[name]["folder"], dtype=dtype, page_size=made[name]["page"],
                                   max_tokens=max_tokens or 512, max_requests=max_requests, max_batched_tokens=256,
                                   max_model_len=256, cuda_graph=graph, check_cache=True)
    return _engines[key]


def load(folder, dtype, page=4, tokens=64, requests=2, longest=64, check=True):
    from fastllm_py_b200 import Model

    return Model.load(folder, dtype=dtype, page_size=page, max_tokens=tokens, max_requests=requests,
                      max_batched_tokens=max(64, longest), max_model_len=longest, cuda_graph=False, check_cache=check).engine


def cuts(requests, live):
    return {"whole": replay.whole(requests), "tail": replay.tail_decode(requests, 12),
            "portions": replay.portions(requests), "small": replay.portions(requests, (2, 3, 2, 5, 2)),
            "mixed": replay.mixed(requests, live=live, seed=3, prefill_sizes=(9, 2, 17, 5), decode_tail=6)}


def worst(got, want):
    return max(float((got[(rid, p)] - want[rid][p]).abs().max()) for (rid, p) in got)


def errors(got, want, spread):
    return np.array([float((got[k] - want[k[0]][k[1]]).pow(2).mean().sqrt()) for k in got]) / spread


@pytest.mark.parametrize("name", list(MODELS))
def test_every_cut_in_32_bit_equals_the_oracle_and_the_other_cuts(made, name):
    m = made[name]
    top = max(float(v.abs().max()) for v in m["want"].values())
    results = {}
    for cut, steps in cuts(m["requests"], live=3).items():
        pool = replay.peak_tokens(steps, m["page"]) + (0 if cut == "mixed" else m["page"])
        eng = engine(made, name, "float32", pool).engine
        got = replay.run_in_process(eng, steps)
        assert len(got) == sum(len(t) for t in m["requests"].values())
        assert worst(got, m["want"]) <= 2e-4 * max(1.0, top), cut
        results[cut] = got
        assert not eng.cache.live
    for cut, got in results.items():
        for key, row in got.items():
            assert torch.equal(row, results["whole"][key]), (cut, key)


@pytest.mark.parametrize("name", list(MODELS))
def test_every_cut_in_bfloat16_stays_near_the_oracle(made, name):
    """Where two experts' scores are a rounding apart the engine may take the other one: a few positions may be far."""
    m = made[name]
    spread = float(torch.cat([v.flatten() for v in m["want"].values()]).std())
    for cut, steps in cuts(m["requests"], live=3).items():
        eng = engine(made, name, "bfloat16", replay.peak_tokens(steps, m["page"]) + m["page"]).engine
        errs = np.sort(errors(replay.run_in_process(eng, steps), m["want"], spread))
        assert np.median(errs) <= 0.04, (cut, np.median(errs))
        assert errs[int(len(errs) * 0.95) - 1] <= 0.15, (cut, errs[-8:])


SMALL = dict(width=24, vocab=50)
LEFT, RIGHT = kt.left(1, 1, 4, 4, rot=2), kt.right(4, 2, 1, 1)
SINGLE = {
    "latent": kt.config([(kt.latent(2, 8, 4, 12, 10, 14), None)], **SMALL),
    "latent_one_head": kt.config([(kt.latent(1, 3, 2, 1, 1, 1), None)], **SMALL),
    "latent_many_heads": kt.config([(kt.latent(19, 4, 16, 8, 32, 24), None)], **SMALL),
    "latent_wide": kt.config([(kt.latent(2, 72, 64, 100, 160, 40), None)], **SMALL),
    "latent_uneven": kt.config([(kt.latent(3, 17, 10, 33, 48, 31), None)], **SMALL),
    "left": kt.config([(kt.pair(kt.left(6, 2, 24, 40, rot=10, factor=5.0), RIGHT, 1.5, 0.1), None)], **SMALL),
    "left_one_value": kt.config([(kt.pair(kt.left(4, 1, 8, 1, rot=8), RIGHT, 1.5, 0.1), None)], **SMALL),
    "left_wide": kt.config([(kt.pair(kt.left(3, 1, 136, 200, rot=30), RIGHT, 1.5, 0.1), None)], **SMALL),
    "left_group_of_twelve": kt.config([(kt.pair(kt.left(12, 1, 16, 16, rot=16), RIGHT, 1.5, 0.1), None)], **SMALL),
    "scan": kt.config([(kt.pair(LEFT, kt.right(40, 16, 8, 4), 0.1, 1.2), None)], **SMALL),
    "scan_one": kt.config([(kt.pair(LEFT, kt.right(1, 1, 1, 1), 0.1, 1.2), None)], **SMALL),
    "scan_many_taps": kt.config([(kt.pair(LEFT, kt.right(24, 20, 5, 11), 0.1, 1.2), None)], **SMALL),
    "scan_state_50": kt.config([(kt.pair(LEFT, kt.right(18, 50, 40, 2), 0.1, 1.2), None)], **SMALL),
    "scan_state_100": kt.config([(kt.pair(LEFT, kt.right(20, 100, 3, 3), 0.1, 1.2), None)], **SMALL),
    "scan_state_256": kt.config([(kt.pair(LEFT, kt.right(17, 256, 2, 3), 0.1, 1.2), None)], **SMALL),
    "scan_rank_wide": kt.config([(kt.pair(LEFT, kt.right(33, 8, 150, 3), 0.1, 1.2), None)], **SMALL),
    "dense": kt.config([(kt.pair(LEFT, RIGHT), kt.dense(36))], **SMALL),
    "experts": kt.config([(kt.pair(LEFT, RIGHT, 0.2, 0.2), kt.moe(12, 4, 20, 0.7))], **SMALL),
    "experts_all": kt.config([(kt.pair(LEFT, RIGHT, 0.2, 0.2), kt.moe(3, 3, 5, 2.0))], **SMALL),
    "loop": kt.config([(kt.pair(LEFT, RIGHT), None), (kt.latent(1, 8, 2, 8, 8, 8), kt.dense(8))], loop=(1, 2, 4), **SMALL),
    "cap": kt.config([(kt.pair(LEFT, RIGHT), None)], cap=0.8, **SMALL),
}


@pytest.mark.parametrize("kind", list(SINGLE))
def test_each_mechanism_alone(tmp_path, kind):
    """A prompt, then single tokens, in both precisions (the bfloat16 engine's fused single-token kernels among them)."""
    from fastllm_py_b200 import StepEntry

    raw = SINGLE[kind]
    w = kt.weights(raw, seed=17)
    folder = kt.write(raw, w, tmp_path / kind)
    toks = np.random.default_rng(1).integers(0, raw["vocab"], size=45).tolist()
    want = plain.forward(raw, w, toks).float()
    for dtype in ("float32", "bfloat16"):
        eng = load(folder, dtype)
        eng.begin("a")
        head = eng.step([StepEntry("a", toks[:20], list(range(20)))]).cpu().clone()
        rest = [eng.step([StepEntry("a", [t], [0])]).cpu().clone() for t in toks[20:]]
        got = torch.cat([head] + rest)
        if dtype == "float32":
            assert float((got - want).abs().max()) <= 2e-4 * max(1.0, float(want.abs().max()))
        else:
            errs = np.sort(((got - want).pow(2).mean(dim=1).sqrt() / want.std()).numpy())
            assert errs[-3] <= 0.1 and np.median(errs) <= 0.05, errs[-5:]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_mechanism_moves_the_logits(tmp_path, dtype):
    """The engine equals the oracle, and the oracle with one reading changed is far from both."""
    raw = kt.config([(kt.pair(kt.left(4, 2, 8, 8, rot=8, scale=1.0), kt.right(20, 6, 4, 3), 0.9, 0.5), kt.dense(16)),
                     (kt.latent(2, 8, 4, 6, 8, 12, scale=1.0), kt.moe(5, 2, 12))], width=24, vocab=30, loop=(0, 2, 2), cap=4.0)
    w = kt.weights(raw, seed=1)
    folder = kt.write(raw, w, tmp_path / "m")
    toks = np.random.default_rng(3).integers(0, 30, size=40).tolist()
    want = plain.forward(raw, w, toks).float()
    got = replay.run_in_process(load(folder, dtype), replay.portions({"a": toks}, (7, 2, 11)))
    rows = torch.stack([got[("a", p)] for p in range(len(toks))])

    def err(other):                                  # middle position's distance of a row, in spreads
        return float((other - rows).pow(2).mean(dim=1).sqrt().median() / want.std())

    base = err(want)
    assert base <= (2e-5 if dtype == "float32" else 0.03), base
    for alter in ALTERS:
        other = err(plain.forward(raw, w, toks, alter={alter}).float())
        assert other > (100 if dtype == "float32" else 2) * base, (alter, other, base)


def _loud_key(raw, kind):
    """Weights under which the vocabulary's last token, as a query, is answered by an earlier token of the one before it and
    by nothing else: the two are the only rows of the embedding that are not zero in the first and in the second quarter
    of the width, and the queries of every head read the first quarter as the keys read the second."""
    w = kt.weights(raw, seed=8)
    width, m = raw["width"], raw["layers"][0]["mixer"]
    quarter = width // 4
    gen = torch.Generator().manual_seed(12)
    w["embed"][:, :2 * quarter] = 0.0
    w["embed"][-2:] = 0.0
    loud = (2.0 + torch.rand(quarter, generator=gen)).to(torch.bfloat16)
    w["embed"][-1, :quarter] = loud
    w["embed"][-2, quarter:2 * quarter] = loud
    w["l0.norm1"] = torch.ones(width, dtype=torch.bfloat16)

    def reads(rows, at):
        block = torch.zeros(rows, width)
        block[:, at * quarter:(at + 1) * quarter] = torch.randn(rows, quarter, generator=torch.Generator().manual_seed(3))
        return block.to(torch.bfloat16)

    if kind == "left":
        m, at = m["left"], "l0.mix.left."
        w[at + "q"], w[at + "k"] = reads(m["dim"], 0).repeat(m["heads"], 1), reads(m["dim"], 1).repeat(m["kv_heads"], 1)
        for s in ("q.norm", "k.norm"):
            w[at + s] = torch.ones_like(w[at + s])
    else:
        at = "l0.mix."
        w[at + "dq"] = reads(m["q_rank"], 0)
        w[at + "dkv"][:m["kv_rank"]] = reads(m["kv_rank"], 1)
        for s in ("dq.norm", "dkv.norm"):
            w[at + s] = torch.ones_like(w[at + s])
        up = (torch.randn(m["dim"], m["kv_rank"], generator=gen) * m["kv_rank"] ** -0.5).to(torch.bfloat16)
        uq = torch.zeros(m["heads"], m["dim"] + m["rot_dim"], m["q_rank"], dtype=torch.bfloat16)
        uq[:, :m["dim"]] = up
        w[at + "uq"] = uq.view(-1, m["q_rank"])
        w[at + "uk"] = up.repeat(m["heads"], 1)
    return w


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["latent", "left"])
def test_a_far_key_among_hundreds_stands_out(tmp_path, dtype, kind):
    """One early token answers a late query among 300 keys (in a prompt, and alone in a decode step, behind page borders);
    without that token the oracle is far away."""
    if kind == "latent":
        mixer = kt.latent(4, 32, 16, 16, 32, 32, scale=0.5)
    else:
        mixer = kt.pair(kt.left(4, 1, 32, 16, rot=4, base=1e6, scale=0.6), kt.right(4, 2, 1, 1), 1.0, 0.05)
    raw = kt.config([(mixer, None)], width=32, vocab=40, scale=1.0, cap=None)
    w = _loud_key(raw, kind)
    folder = kt.write(raw, w, tmp_path / "far")
    toks = np.random.default_rng(5).integers(0, 38, size=300).tolist()
    toks[33] = 38
    eng = load(folder, dtype, page=16, tokens=320, requests=1, longest=320)
    for p in (40, 271, 287):                         # behind a page's border, and the last and first places of pages
        seq = toks[:p] + [39]
        want = plain.forward(raw, w, seq).float()
        without = plain.forward(raw, w, seq[:33] + [0] + seq[34:]).float()
        gap = float((without[p] - want[p]).pow(2).mean().sqrt())
        assert gap > 0.2 * float(want.std())
        for steps in (replay.whole({"a": seq}), replay.tail_decode({"a": seq}, 1), replay.portions({"a": seq}, (64, 30, 2))):
            row = replay.run_in_process(eng, steps)[("a", p)]
            err = float((row - want[p]).pow(2).mean().sqrt())
            assert err <= (1e-4 if dtype == "float32" else 0.05) * float(want.std()) and err < 0.2 * gap


def test_far_tokens_reach_through_the_state(tmp_path):
    """Decays close to one: the first token still moves the last logits through the state alone, and the engine follows
    the oracle through 150 single-token steps after a short prompt, in both precisions."""
    raw = kt.config([(kt.pair(kt.left(1, 1, 4, 4, rot=2), kt.right(40, 16, 4, 3), 0.0, 1.0), kt.dense(16)),
                     (kt.pair(kt.left(1, 1, 4, 4, rot=2), kt.right(24, 5, 3, 4), 0.0, 1.0), None)], width=24, vocab=40, cap=None)
    w = kt.weights(raw, seed=9, slow=True)
    folder = kt.write(raw, w, tmp_path / "far")
    toks = np.random.default_rng(4).integers(0, 40, size=160).tolist()
    want = plain.forward(raw, w, toks).float()
    changed = plain.forward(raw, w, [(toks[0] + 1) % 40] + toks[1:]).float()
    eng = load(folder, "float32", page=16, tokens=256, longest=256, check=False)
    got = replay.run_in_process(eng, replay.tail_decode({"a": toks}, 150))
    err = worst(got, {"a": want})
    assert err <= 2e-4 * float(want.abs().max())
    assert float((changed[-1] - want[-1]).abs().max()) > 30 * max(err, 1e-5)
    eng = load(folder, "bfloat16", page=16, tokens=256, longest=256, check=False)
    got = replay.run_in_process(eng, replay.tail_decode({"a": toks}, 150))
    errs = [float((got[("a", p)] - want[p]).pow(2).mean().sqrt() / want.std()) for p in range(160)]
    assert max(errs[100:]) <= 0.08, max(errs[100:])                      # nothing piles up along the decode


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(2, 8, 4, 12, 10, 14), (3, 16, 16, 16, 32, 16)])
def test_the_sink_takes_most_of_the_weight(tmp_path, dtype, sizes):
    """A sink above every score: a row without it would be several times larger, from the first token on, in prompts and
    in decode steps (sizes of the CUDA-core and of the tensor-core kernel)."""
    raw = kt.config([(kt.latent(*sizes), None)], width=32, vocab=40, cap=None)
    w = kt.weights(raw, seed=4)
    w["l0.mix.sink"] = torch.tensor([4.0, 3.0, 5.0][:sizes[0]], dtype=torch.bfloat16)
    folder = kt.write(raw, w, tmp_path / "sink")
    toks = np.random.default_rng(6).integers(0, 40, size=40).tolist()
    want = plain.forward(raw, w, toks).float()
    without = plain.forward(raw, w, toks, alter={"no_sink"}).float()
    for steps in (replay.whole({"a": toks}), replay.tail_decode({"a": toks}, 39)):
        got = replay.run_in_process(load(folder, dtype), steps)
        for p in range(40):
            err = float((got[("a", p)] - want[p]).pow(2).mean().sqrt())
            assert err <= 0.1 * float((without[p] - want[p]).pow(2).mean().sqrt()), p


def test_a_slot_used_again_starts_clean(made):
    """Two requests one after the other in an engine with a single slot equal the same requests in
    fresh engines, bit for bit (states and kept inputs of the convolutions among them)."""
    m = made["mix"]
    (ra, ta), (rb, tb) = list(m["requests"].items())[3:5]
    eng = engine(made, "mix", "float32", 128, max_requests=1).engine
    first = replay.run_in_process(eng, replay.portions({ra: ta}))
    second = replay.run_in_process(eng, replay.portions({rb: tb}, (1, 1, 1, 2, 7)))
    alone = replay.run_in_process(engine(made, "mix", "float32", 512).engine, replay.whole({rb: tb}))
    assert all(torch.equal(second[k], alone[k]) for k in alone)
    assert worst(first, m["want"]) <= 2e-4 * 30.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_scheduler(made, dtype):
    """Model.generate (scheduler, sampler, captured decode steps, tokens fed on the device) against the oracle's greedy
    loop; where the oracle's two best logits are close the engine may take either."""
    m = made["mix"]
    model = engine(made, "mix", dtype, 512, max_requests=3, graph=True)
    prompts = [m["requests"]["q2"], m["requests"]["q3"], m["requests"]["q1"], m["requests"]["q4"][:20]]
    outs = model.generate(prompts, max_new_tokens=12)
    assert model.generate(prompts, max_new_tokens=12, use_graph=False) == outs          # replayed steps change nothing
    gaps = []                                                    # how far below the oracle's best each token is, in spreads
    for prompt, new in zip(prompts, outs):
        seq = list(prompt)
        for tok in new:
            logits = plain.forward(m["raw"], m["weights"], seq)[-1]
            gaps.append(float(logits.max() - logits[tok]) / float(logits.std()))
            seq.append(tok)
        assert len(new) == 12
    gaps = np.sort(gaps)
    assert gaps[-1] < (1e-3 if dtype == "float32" else 1.0) and gaps[-4] < 0.3, gaps[-5:]


def test_trace_program_on_a_folder(made, tmp_path):
    m = made["odd"]
    steps = replay.mixed(m["requests"], live=2, seed=1, prefill_sizes=(7, 2, 30), decode_tail=3)
    got = replay.run_program(m["folder"], "float32", steps, tmp_path / "out", replay.peak_tokens(steps, 64),
                             m["raw"]["vocab"], extra_args=("--max-requests", "2"))
    top = max(float(v.abs().max()) for v in m["want"].values())
    assert worst(got, m["want"]) <= 2e-4 * max(1.0, top)


def test_command_line_on_a_random_weights_folder(tmp_path):
    """bin/make_model writes a folder from a configuration, bin/generate loads it by its architecture
    string and generates through the scheduler."""
    import json
    import subprocess
    import sys

    raw = kt.config([(kt.latent(2, 16, 16, 16, 32, 32), kt.moe(4, 2, 16)),
                     (kt.pair(kt.left(2, 1, 16, 16), kt.right(32, 16, 4, 4)), kt.dense(32))], width=32, vocab=64, loop=(0, 2, 2))
    (tmp_path / "config.json").write_text(json.dumps(raw))
    made_ = subprocess.run([sys.executable, str(replay.ROOT / "bin" / "make_model"), str(tmp_path / "config.json"),
                            str(tmp_path / "m"), "--seed", "4", "--std", "0.2"], capture_output=True, text=True)
    assert made_.returncode == 0 and "Kerirax" in made_.stdout, made_.stderr
    run = subprocess.run([sys.executable, str(replay.ROOT / "bin" / "generate"), str(tmp_path / "m"), "-", "9",
                          "bfloat16", "--random-prompt", "30", "--seed", "1"], capture_output=True, text=True)
    assert run.returncode == 0, run.stderr[-2000:]
    lines = run.stdout.strip().splitlines()
    assert "Kerirax: 2L width=32" in lines[0]
    assert len([int(t) for t in lines[1].split(",")]) == 9


def drawn_model(rng):
    """A configuration drawn at random: layer kinds in any order, any loop, sizes from lists that hold the awkward ones."""
    ch = rng.choice
    layers = []
    for _ in range(rng.randint(2, 5)):
        if rng.random() < 0.4:
            mixer = kt.latent(ch([1, 2, 3, 5, 16, 17]), ch([4, 8, 15, 32, 64]), ch([2, 8, 16, 32]), ch([4, 9, 16, 48, 80]),
                              ch([8, 20, 32, 64, 96, 128]), ch([8, 12, 33, 64]), ch([500.0, 1e4, 1e6]), ch([None, 0.1, 0.3]))
        else:
            kv, group, dim = ch([1, 2, 3]), ch([1, 1, 2, 3, 4, 12]), ch([8, 12, 16, 24, 32, 48, 64, 72, 128])
            rot = None if rng.random() < 0.15 else ch([dim, 2 * rng.randint(1, dim // 2)])
            l = kt.left(kv * group, kv, dim, ch([4, 8, 24, 32, 48, 100, 128]), rot, ch([500.0, 1e6]), ch([None, 2.0, 8.0]),
                        ch([None, 0.1, 0.3]))
            r = kt.right(ch([8, 12, 20, 33, 64, 96, 136]), ch([1, 4, 12, 16, 32, 50, 64, 128, 200]), ch([1, 3, 8, 16, 33, 72]),
                         ch([1, 2, 3, 4, 4, 5]))
            mixer = kt.pair(l, r, ch([0.6, 1.0, -0.4]), ch([0.5, 1.0, 1.7]))
        f = rng.random()
        experts = ch([1, 4, 9, 16])
        layers.append((mixer, None if f < 0.25 else kt.dense(ch([16, 30, 64, 256])) if f < 0.6 else
                       kt.moe(experts, rng.randint(1, min(experts, 4)), ch([8, 20, 32, 64]), ch([0.8, 2.0, 7.0]))))
    loop = None
    if rng.random() < 0.85:
        start = rng.randint(0, len(layers) - 1)
        loop = (start, rng.randint(start + 1, len(layers)), ch([1, 2, 3]))
    return kt.config(layers, rng.randint(50, 200), ch([24, 40, 64, 136]), ch([1e-5, 1e-6]), loop, ch([0.5, 1.0, 3.0]), ch([None, 5.0, 30.0]))


@pytest.mark.parametrize("seed", [0, 1, 2, 3, 4, 5, 6, 7])
def test_configurations_drawn_at_random(tmp_path, seed):
    import random

    rng = random.Random(seed)
    raw = drawn_model(rng)
    w = kt.weights(raw, seed=seed)
    requests = {f"q{i}": np.random.default_rng(seed + i).integers(0, raw["vocab"], size=n).tolist()
                for i, n in enumerate([rng.randint(1, 45) for _ in range(3)])}
    want = {rid: plain.forward(raw, w, toks).float() for rid, toks in requests.items()}
    folder = kt.write(raw, w, tmp_path / "m")
    steps = replay.mixed(requests, live=2, seed=seed, prefill_sizes=(9, 2, 17, 5), decode_tail=6)
    top = max(float(v.abs().max()) for v in want.values())
    got = replay.run_in_process(load(folder, "float32", page=8, tokens=replay.peak_tokens(steps, 8) + 8), steps)
    assert worst(got, want) <= 2e-4 * max(1.0, top), raw
    got = replay.run_in_process(load(folder, "bfloat16", page=8, tokens=replay.peak_tokens(steps, 8) + 8), steps)
    errs = errors(got, want, float(torch.cat([v.flatten() for v in want.values()]).std()))
    assert np.median(errs) <= 0.06, (np.median(errs), raw)
