"""Kernels of the Kerirax design alone, against the oracle's functions or plain torch, and its parts in other arrangements."""
from types import SimpleNamespace

import pytest
import torch

import plain_kerirax as plain
from test_lufozen_kernels_gpu import LENS, SCHEDULE, dev, i32, step_of

pytestmark = pytest.mark.gpu


def near(got, ref, tol, what=None):
    assert float((got.double().cpu() - ref).abs().max()) <= tol * max(1.0, float(ref.abs().max())), what


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes,pad", [((40, 16, 8, 4), 0), ((40, 16, 8, 4), 1), ((13, 1, 1, 1), 0), ((96, 30, 20, 3), 4), ((24, 64, 72, 2), 0),
                                       ((20, 100, 5, 9), 0), ((17, 256, 33, 4), 3), ((132, 9, 16, 16), 0), ((8, 32, 12, 4), 0)])
def test_selective_scan_kernels_over_steps(dtype, sizes, pad):
    """inner, state, rank, taps; columns of something else before and behind the rows and `pad` floats behind a state row, so
    that wide and narrow accesses both run; steps of single tokens also through the one-kernel form."""
    from fastllm_py_b200.native import ops

    inner, N, rank, taps = sizes
    gen = torch.Generator().manual_seed(sum(sizes))

    def r(*shape, std=1.0):
        return torch.randn(*shape, generator=gen) * std

    proj = [r(n, 2 * inner).to(dtype) for n in LENS]
    m = {"inner": inner, "state": N, "dt_rank": rank, "conv": taps}
    t = {"in": torch.eye(2 * inner), "conv": r(inner, taps, std=0.6), "conv.b": r(inner, std=0.3),
         "x": r(rank + 2 * N, inner, std=inner ** -0.5), "dt": r(inner, rank, std=rank ** -0.5).bfloat16(), "dt.b": r(inner) - 2.0,
         "A_log": r(inner, N, std=0.6), "D": r(inner), "o": torch.eye(inner)}
    t = {k: v.double() for k, v in t.items()}
    want = [plain.selective_scan(p.double(), t, m)[0] * 0.7 for p in proj]
    f32 = lambda v: dev(v.float().contiguous())
    conv_w, conv_b, bias, skip, w_x, w_dt = f32(t["conv"].T), f32(t["conv.b"]), f32(t["dt.b"]), f32(t["D"]), f32(t["x"]), f32(t["dt"])
    wide = torch.zeros(inner, -(-rank // 8) * 8, dtype=torch.bfloat16, device="cuda")
    wide[:, :rank] = w_dt
    a = -torch.exp(t["A_log"])
    a = f32(a * 1.4426950408889634 if dtype == torch.bfloat16 else a)
    floats = -(-inner * N // 4) * 4
    for fused in (False, True):
        state = torch.full((3, floats + (taps - 1) * inner + pad), 1e4, device="cuda")
        tail = state[:, floats:] if taps > 1 else None
        for entries in SCHEDULE:
            step, starts = step_of(entries, {0: 2, 1: 0})
            n = step.n_tokens
            p = torch.full((n, 2 * inner + 16), 7.0, dtype=dtype, device="cuda")
            p[:, 8:8 + 2 * inner] = dev(torch.cat([proj[q][b:b + c] for q, b, c in entries]))
            u, z = p[:, 8:8 + inner], p[:, 8 + inner:8 + 2 * inner]
            x = torch.empty(n, inner, dtype=dtype, device="cuda")
            y = torch.empty(n, inner + 8, dtype=dtype, device="cuda")[:, :inner]
            single = fused and n == step.n_requests
            ops.selective_conv(u, conv_w, conv_b, tail, step, x, single)
            low = x.float() @ w_x.T                                   # (torch: the products are not what is tested)
            if single:
                ops.selective_step(x, z, low, rank, wide, bias, a, skip, 0.7, y, state, step)
            else:
                dt = low[:, :rank] @ w_dt.T
                if dtype == torch.bfloat16:
                    parts = torch.empty(n, 2 * rank, dtype=dtype, device="cuda")
                    ops.selective_split(low, rank, parts)
                    near(parts[:, :rank].double() + parts[:, rank:].double(), low[:, :rank].double().cpu(), 2e-5)
                    dt = (parts.float() @ torch.cat([w_dt, w_dt], 1).T)
                ops.selective_scan(x, z, u, dt.contiguous(), bias, low, rank, a, skip, 0.7, y, state, floats, taps, step)
            for i, (q, b, c) in enumerate(entries):
                near(y[starts[i]:starts[i + 1]], want[q][b:b + c], 2e-4 if dtype == torch.float32 else 0.06, (entries, q, fused))
        assert float(state[1].min()) == 1e4                                  # a slot of no request is left alone


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_convolution_of_long_steps(dtype, taps):
    """Steps in which a thread takes several tokens, runs that end with a request or with the step among them."""
    from fastllm_py_b200.native import ops

    inner = 20
    gen = torch.Generator().manual_seed(taps)
    w, b = torch.randn(inner, taps, generator=gen) * 0.6, torch.randn(inner, generator=gen) * 0.3
    for lengths in ((300,), (259, 6), (1101,), (3, 1030, 2)):
        u = [torch.randn(n, inner, generator=gen).to(dtype) for n in lengths]
        tails = torch.randn(len(lengths), (taps - 1) * inner, generator=gen)
        ctx = [0 if i % 2 else 50 for i in range(len(lengths))]
        step, starts = step_of([(i, ctx[i], n) for i, n in enumerate(lengths)], {i: i for i in range(len(lengths))})
        kept = dev(tails) if taps > 1 else None
        x = torch.empty(sum(lengths), inner, dtype=dtype, device="cuda")
        ops.selective_conv(dev(torch.cat(u)), dev(w.T.contiguous()), dev(b), kept, step, x, False)
        for i, n in enumerate(lengths):
            tail = tails[i].view(taps - 1, inner).double() * (1.0 if ctx[i] else 0.0)
            want = plain.silu(plain.short_conv(u[i].double(), w.double(), b.double(), tail))
            near(x[starts[i]:starts[i + 1]], want, 1e-5 if dtype == torch.float32 else 0.01, (lengths, i))


def test_the_scan_is_the_same_whatever_the_cut_and_the_batch():
    """32-bit: one order of sums, bit for bit, alone and beside seven other requests, whole and in portions."""
    from fastllm_py_b200.native import ops

    inner, N, rank, taps, T = 36, 20, 4, 4, 150
    gen = torch.Generator(device="cuda").manual_seed(1)
    r = lambda *s: torch.randn(*s, device="cuda", generator=gen)
    x, z, u, dt, low = r(T, inner), r(T, inner), r(T, inner), r(T, inner) - 2, r(T, rank + 2 * N)
    a, skip, bias = -torch.rand(inner, N, device="cuda"), r(inner), r(inner)

    def run(pieces, others):
        state = torch.zeros(1 + others, inner * N + (taps - 1) * inner, device="cuda")
        outs, at = [], 0
        for c in pieces:
            sl = slice(at, at + c)
            # the request itself stands last in the batch
            entries = [(k + 1, at, c) for k in range(others)] + [(0, at, c)]
            step, starts = step_of(entries, {k: k for k in range(others + 1)})
            cat = lambda v: torch.cat([torch.roll(v, k + 1, 0)[sl] for k in range(others)] + [v[sl]])
            y = torch.empty(step.n_tokens, inner, device="cuda")
            ops.selective_scan(cat(x), cat(z), cat(u), cat(dt), bias, cat(low), rank, a, skip, 1.0, y, state, inner * N, taps, step)
            outs.append(y[starts[others]:starts[others + 1]].clone())
            at += c
        return torch.cat(outs), state[0].clone()

    whole, end = run([T], 0)
    for pieces in ([1] * T, [2, 15, 16, 17, 100], [64, 64, 22], [149, 1]):
        for others in (0, 7):
            y, s = run(pieces, others)
            assert torch.equal(y, whole) and torch.equal(s, end), (pieces, others)


def test_a_long_sequence_does_not_drift():
    """6000 tokens of decays within 1e-3 of one: the 32-bit scan's state stays a few roundings from float64's."""
    from fastllm_py_b200.native import ops

    inner, N, rank, T = 8, 8, 1, 6000
    gen = torch.Generator().manual_seed(2)
    x = torch.rand(T, inner, generator=gen) + 0.5
    low = torch.rand(T, rank + 2 * N, generator=gen)
    dt = torch.full((T, inner), -7.0) + 0.3 * torch.randn(T, inner, generator=gen)
    a = -torch.rand(inner, N, generator=gen) - 0.2
    S, d = torch.zeros(inner, N, dtype=torch.float64), torch.nn.functional.softplus(dt.double())
    for i in range(T):
        S = torch.exp(d[i][:, None] * a.double()) * S + (d[i] * x[i].double())[:, None] * low[i, rank:rank + N].double()
    state = torch.zeros(1, inner * N, device="cuda")
    step, _ = step_of([(0, 0, T)], {0: 0})
    y = torch.empty(T, inner, device="cuda")
    ops.selective_scan(dev(x), dev(x), dev(x), dev(dt), torch.zeros(inner, device="cuda"), dev(low), rank, dev(a),
                       torch.zeros(inner, device="cuda"), 1.0, y, state, inner * N, 1, step)
    rel = (state[0].view(inner, N).double().cpu() - S).abs() / S.abs()
    assert float(rel.max()) < 5e-6, float(rel.max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes,rot,interleaved", [((4, 2, 16, 24), 16, True), ((4, 2, 16, 24), 6, True), ((3, 1, 128, 128), 128, False),
                                                   ((3, 3, 10, 7), 6, True), ((12, 1, 72, 1), 20, False), ((2, 2, 64, 8), 0, False)])
def test_preparation_with_norms_over_the_whole_projection(dtype, sizes, rot, interleaved):
    from fastllm_py_b200.native import ops

    H, G, d, dv = sizes
    gen = torch.Generator().manual_seed(sum(sizes))
    n, page, eps = 37, 8, 1e-5
    cols = (H + G) * d + G * dv
    proj = torch.randn(n, cols + 8, generator=gen).to(dtype)
    bias = torch.randn(cols, generator=gen) * 0.3
    q_w, k_w = 1 + 0.3 * torch.randn(H * d, generator=gen), 1 + 0.3 * torch.randn(G * d, generator=gen)
    pos = torch.randint(0, 300, (n,), generator=gen)
    slots = torch.randperm(64, generator=gen)[:n].to(torch.int32)
    spec = {"dims": rot, "base": 700.0, "scaling": {"factor": 3.0}}
    cos = sin = None
    if rot:
        ang = torch.arange(300, dtype=torch.float64)[:, None] * plain.rotary_frequencies(rot, 700.0, spec["scaling"])[None, :]
        cos, sin = dev(torch.cos(ang).float()), dev(torch.sin(ang).float())
    for b in (None, bias):
        u = proj[:, :cols].double() + (0.0 if b is None else b.double())
        q = (plain.rms(u[:, :H * d], eps) * q_w.double()).view(n, H, d)
        k = (plain.rms(u[:, H * d:(H + G) * d], eps) * k_w.double()).view(n, G, d)
        if rot:
            pairing = "interleaved" if interleaved else "half"
            q = torch.cat([plain.rotate(q[i:i + 1], spec, int(pos[i]), pairing) for i in range(n)])
            k = torch.cat([plain.rotate(k[i:i + 1], spec, int(pos[i]), pairing) for i in range(n)])
        v = u[:, (H + G) * d:].view(n, G, dv) * 0.6
        cache = torch.full((8, G, page, d + dv), 5.0, dtype=dtype, device="cuda")
        out = torch.empty(n, H * d, dtype=dtype, device="cuda")
        ops.sink_prep(dev(proj)[:, :cols], None if b is None else dev(b), dev(q_w), dev(k_w), eps, out, H, G, d, dv, 0, 0.0, None,
                      dev(slots), cache, page, rot, interleaved, cos, sin, dev(pos.to(torch.int32)), 0.6)
        tol = 2e-6 if dtype == torch.float32 else 0.01
        near(out.view(n, H, d), q, tol)
        rows = cache.permute(0, 2, 1, 3).reshape(64, G, d + dv)
        near(rows[slots.long()][..., :d], k, tol)
        near(rows[slots.long()][..., d:], v, tol)
        other = torch.ones(64, dtype=torch.bool)
        other[slots.long()] = False
        assert float((rows[dev(other)] - 5.0).abs().max()) == 0.0                # rows of no token are left alone


@pytest.mark.parametrize("kernel", ["simt", "tc", "decode"])
def test_one_gate_a_head_in_every_attention_kernel(kernel):
    from fastllm_py_b200.native import ops

    H, G, d, dv, page, T = 4, 2, 32, 48, 16, 70
    gen = torch.Generator().manual_seed(3)
    q, k, v = torch.randn(T, H, d, generator=gen), torch.randn(T, G, d, generator=gen), torch.randn(T, G, dv, generator=gen)
    gate = torch.randn(T, H + 3, generator=gen).bfloat16()[:, 3:]
    q, k, v = q.bfloat16(), k.bfloat16(), v.bfloat16()
    want = plain.softmax_attention(q.double(), k.double(), v.double(), 0.2) * torch.sigmoid(gate.double())[:, :, None]
    cache = torch.zeros(6, G, page, d + dv, dtype=torch.bfloat16, device="cuda")
    for t in range(T):
        cache[t // page, :, t % page, :d], cache[t // page, :, t % page, d:] = dev(k[t]), dev(v[t])
    bt = i32(0, 1, 2, 3, 4, 5).view(1, 6)
    args = (H, G, d, dv, None, 0, 0.2, None, None, None, None, page)
    out = torch.zeros(T, H * dv, dtype=torch.bfloat16, device="cuda")
    qd, gd = dev(q.reshape(T, H * d)), dev(gate)
    step, _ = step_of([(0, 0, T)], {0: 0})
    if kernel == "simt":
        ops.sink_attention_simt(qd, out, cache, bt, step.tok_req, step.positions, *args, gate=gd)
    elif kernel == "tc":
        ops.sink_attention_tc(qd, out, cache, bt, step, *args, gate=gd)
    else:                                            # every token as the single token of a request of its own
        n, kept = ops.sink_decode_splits(None, 0, T)
        part = torch.empty(T * H * n * (dv + 2), device="cuda")
        ops.sink_decode(qd, out, cache, bt.expand(T, 6).contiguous(), i32(*range(T)), step.positions, i32(*range(T)), part, n, kept, *args,
                        gate=gd)
    near(out.view(T, H, dv), want, 0.02)


@pytest.mark.parametrize("n,width,ff,experts,top", [(3, 40, 12, 5, 2), (200, 64, 32, 4, 3), (90, 96, 64, 7, 2)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_experts_weighted_on_their_input(dtype, n, width, ff, experts, top):
    """Few tokens and many (the grouped path in bfloat16), against the oracle's experts for the choice the kernel made."""
    from fastllm_py_b200.parts import BuildContext, PartSpec, build_part
    from fastllm_py_b200.parts.base import Workspace

    gen = torch.Generator().manual_seed(n)
    names = ["router"] + [f"{s}.{e}" for e in range(experts) for s in ("gate", "up", "down")]
    spec = PartSpec("routed_experts", dict(hidden_size=width, experts=experts, top=top, expert_ff=ff, activation="clamped_swish",
                                           activation_params=(0.8, 1.702), weight_on="input", choice_bias=False), {s: s for s in names})
    part = build_part("feed_forward", spec, BuildContext(torch.device("cuda"), dtype, 16, 64))
    w = {k: (torch.randn(*s, generator=gen) * 1.5 * s[1] ** -0.5).bfloat16() for k, s in part.weight_shapes().items()}
    part.load({k: dev(v) for k, v in w.items()})
    h = torch.randn(n, width, generator=gen).to(dtype)
    out = torch.empty(n, width, dtype=dtype, device="cuda")
    part.forward(dev(h), out, SimpleNamespace(workspace=Workspace(torch.device("cuda"), n), n_tokens=n))
    t = {"router": w["router"].double()}
    for e in range(experts):
        t.update({f"e{e}.{s}": w[f"{s}.{e}"].double() for s in ("gate", "up", "down")})
    m = {"router": {"top": top}, "expert": {"limit": 0.8}}
    want, moved = plain.routed_experts(h.double(), t, m), plain.routed_experts(h.double(), t, m, alter={"weight_on_output"})
    near(out, want, 1e-5 if dtype == torch.float32 else 0.03)
    assert float((moved - want).abs().max()) > 0.1


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [40, 33, 2048])
def test_sums_that_wait_are_added_by_the_norm_and_by_the_entrys_operand(dtype, width):
    """x + two pending sums (tensors or slabs of partial sums, or none) + row vectors, in the norm of the stream, gathered or
    not, and as a product's operand."""
    from fastllm_py_b200.native import ops

    gen = torch.Generator(device="cuda").manual_seed(width)
    r = lambda *s: torch.randn(*s, device="cuda", generator=gen)
    n, eps = 9, 1e-5
    x0, w = r(n, width), 1 + 0.3 * r(width)
    ld = -(-width // 4) * 4
    slabs = r(3, n, ld)
    part = SimpleNamespace(data=slabs, ld=ld, splits=3, split_stride=n * ld, check=lambda: None)
    summed = slabs[:, :, :width].double().sum(0)
    t1, t2, vec = r(n, width).to(dtype), r(n, width).to(dtype), r(width)
    cases = [(t1, t2, ()), (part, t2, (vec,)), (t1, part, ()), (None, None, (vec,)), (part, None, (vec, vec)), (None, None, ())]
    rows = i32(7, 0, 7)
    for d1, d2, vectors in cases:
        total = x0.double()
        for d in (d1, d2):
            total = total + (0.0 if d is None else summed if d is part else d.double())
        for v in vectors:
            total = total + v.double()
        want = (total / torch.sqrt((total ** 2).mean(1, keepdim=True) + eps) * w.double()).cpu()
        out, few, operand = (torch.empty(k, width, dtype=dtype, device="cuda") for k in (n, 3, n))
        tol = 1e-5 if dtype == torch.float32 else 0.01
        x = x0.clone()
        ops.norm_pair(x, d1, d2, w, None, few, None, eps, rows, vectors)
        near(few, want[rows.cpu().long()], tol)
        ops.sum_rows(x, d1, d2, operand, vectors)
        near(operand, total.cpu(), tol)
        assert torch.equal(x, x0)                                            # neither moved the stream
        ops.norm_pair(x, d1, d2, w, None, out, None, eps, None, vectors)
        near(out, want, tol)
        near(x, total.cpu(), 1e-6)


def test_parallel_layers_of_other_designs_take_the_new_parts(tmp_path):
    """A scan alone as a mixer, under a norm of its own for the feed-forward, in a pre-norm layer, and a normed pair of two:
    prompts against single tokens in 32-bit, bit for bit."""
    from fastllm_py_b200.parts import BuildContext, Decoder, LayerRun, LayerSpec, ModelPlan, PartSpec
    from fastllm_py_b200 import EngineConfig, StepEntry
    from fastllm_py_b200.engine.engine import Engine

    width = 24
    io = dict(vocab_size=20, hidden_size=width)

    def norm(name):
        return PartSpec("rmsnorm", dict(size=width, eps=1e-5), {"weight": name})

    def scan(at, inner=16, state=6):
        slots = ("in", "conv", "conv_bias", "x", "dt", "dt_bias", "A_log", "D", "o")
        return PartSpec("selective_scan", dict(hidden_size=width, inner=inner, state=state, rank=3, taps=3), {s: at + s for s in slots})

    ff = PartSpec("swiglu", dict(hidden_size=width, intermediate_size=16), {s: "ff." + s for s in ("gate", "up", "down")})
    both = PartSpec("side_by_side", dict(hidden_size=width, left=scan("c."), right=scan("d.", 9, 2), norm_eps=1e-5),
                    {"left_out": "lo", "right_out": "ro"})
    layers = [LayerSpec("parallel", scan("a."), ff, {"mixer": norm("n1"), "feed_forward": norm("n2")}),
              LayerSpec("prenorm", scan("b.", 12, 40), None, {"mixer": norm("n3")}),
              LayerSpec("parallel", both, None, {"mixer": norm("n4")})]
    plan = ModelPlan(hidden_size=width, vocab_size=20, max_positions=64, embedding=PartSpec("table", io, {"weight": "e"}), layers=layers,
                     order=[LayerRun(0), LayerRun(1, entry=True), LayerRun(2), LayerRun(0)], final_norm=norm("n5"),
                     head=PartSpec("linear", io, {"weight": "h"}), entry=PartSpec("rejoin", dict(hidden_size=width), {"weight": "j"}))
    for dtype in ("float32", "bfloat16"):
        dec = Decoder(plan, BuildContext(torch.device("cuda"), getattr(torch, dtype), 4, 64))
        gen = torch.Generator().manual_seed(0)
        dec.load({k: dev((torch.randn(*s, generator=gen) * (0.5 if len(s) > 1 else 0.3) + (1.0 if k.startswith("n") else 0.0)).bfloat16())
                  for k, s in dec.expected_tensors().items()})
        eng = Engine(dec, EngineConfig(dtype=dtype, page_size=4, max_tokens=64, max_requests=2, max_batched_tokens=64, cuda_graph=False), 64, 16)
        toks = torch.randint(0, 20, (30,), generator=gen).tolist()
        eng.begin("a")
        whole = eng.step([StepEntry("a", toks, list(range(30)))]).cpu().clone()
        eng.end("a")
        eng.begin("a")
        alone = torch.cat([eng.step([StepEntry("a", [t], [0])]).cpu().clone() for t in toks])
        assert float(whole.std()) > 0.01
        if dtype == "float32":
            assert torch.equal(whole, alone)
        else:
            assert float((whole - alone).pow(2).mean().sqrt()) <= 0.05 * float(whole.std())
