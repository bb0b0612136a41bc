"""Kernels of the Lufozen design alone, against the oracle's functions or plain torch, and its parts in other arrangements."""
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import lufozen_tiny as lt
import plain_lufozen as plain
import replay

pytestmark = pytest.mark.gpu


def dev(t):
    return t.cuda()


def i32(*v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def step_of(entries, slots):
    """entries: (request, first position, tokens) in the order of the batch; slots: request -> state row."""
    starts = [0]
    for e in entries:
        starts.append(starts[-1] + e[2])
    return SimpleNamespace(
        tok_req=i32(*sum(([i] * e[2] for i, e in enumerate(entries)), [])),
        positions=i32(*sum((list(range(e[1], e[1] + e[2])) for e in entries), [])),
        req_start=i32(*starts), req_ctx=i32(*(e[1] for e in entries)), req_qlen=i32(*(e[2] for e in entries)),
        req_slot=i32(*(slots[e[0]] for e in entries)), n_requests=len(entries), n_tokens=starts[-1],
        n_decode_tokens=sum(e[2] == 1 for e in entries)), starts


# request 0 in slot 2 from the first step; request 1 joins at the third in slot 0; both through single tokens, alone and
# beside portions, through portions shorter and longer than a convolution reaches
SCHEDULE = [[(0, 0, 9)], [(0, 9, 1)], [(0, 10, 1), (1, 0, 11)], [(1, 11, 1), (0, 11, 1)], [(1, 12, 2), (0, 12, 13)], [(0, 25, 1), (1, 14, 1)],
            [(0, 26, 300)], [(1, 15, 260), (0, 326, 2)]]
LENS = [328, 275]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes,pad", [((4, 8, 12, 2, 4, 2), 1), ((4, 8, 12, 2, 4, 2), 4), ((6, 5, 7, 3, 1, 1), 1), ((2, 64, 128, 1, 3, 2), 4),
                                       ((3, 20, 33, 3, 6, 4), 1), ((4, 12, 16, 1, 6, 4), 4), ((1, 7, 200, 1, 2, 1), 1)])
def test_state_space_kernels_over_steps(dtype, sizes, pad):
    """heads, vdim, state, groups, taps, norm parts; a step of single tokens also through the one-kernel form.  `pad`: floats
    behind a state row (four: rows stay on 16 bytes, for the kernels' wide loads)."""
    from fastllm_py_b200.native import ops

    H, P, N, G, taps, parts = sizes
    gen = torch.Generator().manual_seed(sum(sizes))
    inner, ch = H * P, H * P + 2 * G * N
    cols = inner + ch + H
    proj = [torch.randn(n, cols, generator=gen).to(dtype) for n in LENS]
    m = {"heads": H, "vdim": P, "state": N, "groups": G, "conv": taps, "norm_groups": parts if inner % parts == 0 else 1}
    t = {"in": torch.eye(cols), "conv": torch.randn(ch, taps, generator=gen) * 0.6, "conv.b": torch.randn(ch, generator=gen) * 0.3,
         "dt_bias": torch.randn(H, generator=gen) - 2.0, "A_log": torch.randn(H, generator=gen) * 0.5, "D": torch.randn(H, generator=gen),
         "norm": 1 + 0.3 * torch.randn(inner, generator=gen), "o": torch.eye(inner)}
    t = {k: v.double() for k, v in t.items()}
    want = [plain.state_space(p.double(), t, m, 1e-5)[0] for p in proj]
    f32 = lambda v: dev(v.float().contiguous())
    conv_w, conv_b, dt_bias, skip, norm = f32(t["conv"].T), f32(t["conv.b"]), f32(t["dt_bias"]), f32(t["D"]), f32(t["norm"])
    neg_a = dev(-torch.exp(t["A_log"]))
    floats = inner * N
    for fused in (False, True):
        state = torch.full((3, floats + (taps - 1) * ch + pad), 1e4, device="cuda")
        tail = state[:, floats:] if taps > 1 else None
        for entries in SCHEDULE:
            step, starts = step_of(entries, {0: 2, 1: 0})
            n = step.n_tokens
            p = dev(torch.cat([proj[r][a:a + q] for r, a, q in entries]))
            y = torch.empty(n, inner, device="cuda")
            out = torch.empty(n, inner, dtype=dtype, device="cuda")
            if fused and n == step.n_requests:
                ops.ssd_step(p, conv_w, conv_b, dt_bias, neg_a, skip, y, state, floats, step, H, P, N, G)
            else:
                work = torch.empty(n, ch + 2 * H, device="cuda")
                ops.ssd_prep(p, conv_w, conv_b, dt_bias, neg_a, tail, step, work, H, P, N, G)
                ops.ssd_scan(work, skip, y, state, step, H, P, N, G)
            ops.ssd_norm(y, p, norm, out, m["norm_groups"], 1e-5, tail, taps, ch, step)
            for i, (r, a, q) in enumerate(entries):
                got, ref = out[starts[i]:starts[i + 1]].double().cpu(), want[r][a:a + q]
                tol = 1e-4 if dtype == torch.float32 else 0.02
                assert float((got - ref).abs().max()) <= tol * max(1.0, float(ref.abs().max())), (entries, r)
        assert float(state[1].min()) == 1e4                                  # a slot of no request is left alone


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes,taps,rot,pairing,mode", [
    ((4, 2, 16, 24), 4, 8, "interleaved", 1), ((3, 1, 128, 128), 3, 128, "interleaved", 1), ((3, 3, 10, 7), 2, 6, "half", 1),
    ((2, 1, 128, 96), 4, 128, "half", 2), ((2, 2, 48, 64), None, 48, "half", 1), ((2, 1, 72, 36), 1, 72, "interleaved", 1),
    ((1, 1, 200, 140), 4, 100, "half", 0), ((5, 1, 12, 9), 8, 12, "interleaved", 1), ((1, 1, 300, 8), 5, 300, "interleaved", 1)])
def test_convolved_head_preparation_over_steps(dtype, sizes, taps, rot, pairing, mode):
    from fastllm_py_b200.native import ops

    H, G, d, dv = sizes
    gen = torch.Generator().manual_seed(sum(sizes))
    page, ch = 8, (H + G) * d + G * dv
    proj = [torch.randn(n, ch + 5, generator=gen).to(dtype) for n in LENS]       # (five columns of something else behind)
    bias = torch.randn(ch, generator=gen) * 0.4
    conv = None if taps is None else torch.randn(ch, taps, generator=gen) * 0.6
    q_w, k_w = 1 + 0.3 * torch.randn(d, generator=gen), 1 + 0.3 * torch.randn(d, generator=gen)
    spec = {"dims": rot, "base": 300.0}
    ang = torch.arange(400, dtype=torch.float64)[:, None] * plain.rotary_frequencies(rot, 300.0)[None, :]
    cos, sin = dev(torch.cos(ang).float()), dev(torch.sin(ang).float())
    want = []
    for p in proj:
        u = p[:, :ch].double() + bias.double()
        if conv is not None:
            u = plain.short_conv(u, conv.double())
        q, k, v = u[:, :H * d].view(-1, H, d), u[:, H * d:(H + G) * d].view(-1, G, d), u[:, (H + G) * d:].view(-1, G, dv) * 0.7
        if mode == 1:
            q, k = plain.rms(q, 1e-5) * q_w.double(), plain.rms(k, 1e-5) * k_w.double()
        q, k = plain.rotate(q, spec, pairing), plain.rotate(k, spec, pairing)
        if mode == 2:
            q, k = plain.rms(q, 1e-5), plain.rms(k, 1e-5)
        want.append((q.reshape(q.shape[0], -1), k, v))
    back = (taps or 1) - 1
    tail = torch.full((3, max(back * ch, 1)), 1e4, device="cuda")
    cache = torch.zeros(100, G, page, d + dv, dtype=dtype, device="cuda")
    base = {0: 0, 1: 400}                                                        # a request's cache rows, one after another
    w = None if conv is None else dev(conv.T.contiguous())
    tol = 2e-5 if dtype == torch.float32 else 0.02
    for entries in SCHEDULE:
        step, starts = step_of(entries, {0: 2, 1: 0})
        p = dev(torch.cat([proj[r][a:a + n] for r, a, n in entries]))
        slots = i32(*sum((list(range(base[r] + a, base[r] + a + n)) for r, a, n in entries), []))
        q_out = torch.empty(step.n_tokens, H * d, dtype=dtype, device="cuda")
        ops.conv_head_prep(p, dev(bias), w, tail if back else None, dev(q_w) if mode == 1 else None, dev(k_w) if mode == 1 else None,
                           mode, 1e-5, rot, pairing == "interleaved", cos, sin, step, None, 0.7, q_out, H, G, d, dv, slots, cache, page)
        for i, (r, a, n) in enumerate(entries):
            q, k, v = (x[a:a + n] for x in want[r])
            rows = torch.arange(base[r] + a, base[r] + a + n)
            stored = cache[(rows // page).cuda(), :, (rows % page).cuda()].double().cpu()        # [n, G, d + dv]
            for got, ref in ((q_out[starts[i]:starts[i + 1]].double().cpu(), q), (stored[..., :d], k), (stored[..., d:], v)):
                assert float((got - ref).abs().max()) <= tol * max(1.0, float(ref.abs().max())), (entries, r)
    assert float(tail[1].min()) == 1e4


@pytest.mark.parametrize("sizes", [(2, 12, 20), (1, 64, 128), (3, 40, 33), (2, 100, 16), (1, 250, 70)])
def test_scan_with_a_decay_per_row_over_steps(sizes):
    """Bit for bit the same whatever the cut; few and many requests at once."""
    from fastllm_py_b200.native import ops

    H, d, dv = sizes
    gen = torch.Generator().manual_seed(d)
    hd, hv, L = H * d, H * dv, 61
    work = torch.randn(L, 3 * hd + hv, generator=gen)
    work[:, 2 * hd:3 * hd] = torch.rand(L, hd, generator=gen) * 0.3 + 0.7
    q, k, a, v = (work[:, :hd].view(L, H, d).double(), work[:, hd:2 * hd].view(L, H, d).double(),
                  work[:, 2 * hd:3 * hd].view(L, H, d).double(), work[:, 3 * hd:].view(L, H, dv).double())
    S, want = torch.zeros(H, d, dv, dtype=torch.float64), torch.zeros(L, hv, dtype=torch.float64)
    for i in range(L):
        S = a[i][:, :, None] * S + k[i][:, :, None] * v[i][:, None, :]
        want[i] = torch.einsum("hdv,hd->hv", S, q[i]).reshape(-1)
    results = []
    for many in (1, 40, 700):
        for cut in ((L,), (1, 1, 5, 20, 34), (17, 1, 43)):
            state = torch.full((many, H * dv * d), 1e4, device="cuda")
            at, outs = 0, []
            for n in cut:
                entries = [(r, at, n) for r in range(many)]
                step, starts = step_of(entries, {r: many - 1 - r for r in range(many)})
                rows = dev(work[at:at + n].repeat(many, 1))
                o = torch.empty(n * many, hv, device="cuda")
                ops.gla_scan(rows, o, state, step, H, d, dv)
                o = o.view(many, n, hv)
                assert torch.equal(o[0], o[-1])
                outs.append(o[0].cpu())
                at += n
            got = torch.cat(outs)
            assert float((got.double() - want).abs().max()) <= 2e-5 * float(want.abs().max())
            results.append(got)
    assert all(torch.equal(r, results[0]) for r in results)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norms_add_row_vectors_with_what_is_pending(dtype):
    """x += pending + vectors, then the norm: a tensor pending, split-K partial sums, gathered rows, nothing pending."""
    from fastllm_py_b200.native import ops
    from fastllm_py_b200.parts import BuildContext, PartSpec, ResidualStream, build_part

    gen = torch.Generator().manual_seed(1)
    for rows, width in ((19, 44), (3, 1000), (5, 37), (2, 9000)):
        norm = build_part("norm", PartSpec("rmsnorm", dict(size=width, eps=1e-5, offset=1.0, gain=0.5), {"weight": "w"}),
                          BuildContext(torch.device("cuda"), dtype, 8, 8))
        w = (torch.randn(width, generator=gen) * 0.3).to(torch.bfloat16)
        norm.load({"weight": dev(w)})
        x0, d = torch.randn(rows, width, generator=gen) * 3, torch.randn(rows, width, generator=gen).to(dtype)
        vecs = [torch.randn(width, generator=gen) for _ in range(3)]

        class Partial:                                   # what a product with its K split leaves
            splits, split_stride, ld, rows_, cols = 3, rows * (-(-width // 4) * 4), -(-width // 4) * 4, rows, width
            data = torch.zeros(3, rows, -(-width // 4) * 4)

            def check(self):
                pass
        part = Partial()
        part.data[:, :, :width] = d.float()[None] * torch.tensor([0.5, 0.25, 0.25])[:, None, None]
        part.data = dev(part.data)
        tol = 1e-5 if dtype == torch.float32 else 0.02
        for count in (0, 1, 2, 3):
            for pending in ("tensor", "partial", "rows", None):
                stream = ResidualStream(dev(x0.clone()))
                for v in vecs[:count]:
                    stream.add_vector(dev(v))
                stream.pending = {"tensor": dev(d), "rows": dev(d), "partial": part, None: None}[pending]
                total = x0.double() + sum((v.double() for v in vecs[:count]), torch.zeros(width).double())
                if pending is not None:
                    total = total + d.double()
                pick = i32(rows - 1, 0) if pending == "rows" else None
                out = torch.empty(rows if pick is None else 2, width, dtype=dtype, device="cuda")
                stream.norm_into(norm, out, pick)
                ref = total if pick is None else total[[rows - 1, 0]]
                ref = plain.rms(ref, 1e-5) * (1.0 + w.double()) * 0.5
                assert float((out.double().cpu() - ref).abs().max()) <= 2 * tol, (rows, width, count, pending)
                if pick is None:
                    assert float((stream.x.double().cpu() - total).abs().max()) <= 1e-5 * float(total.abs().max()) + (0 if dtype == torch.float32 else 0.02)
                    assert stream.pending is None and stream.vectors == ()
        x = dev(d)
        ops.add_bias(x, dev(vecs[0]))
        assert float((x.double().cpu() - d.double() - vecs[0].double()).abs().max()) <= 2 * tol


def test_products_with_an_activation_on_the_way_out():
    """Few and many rows (K split, one tile, tile pairs) against the product and the activation apart."""
    from fastllm_py_b200.native import gemm_tc

    gen = torch.Generator().manual_seed(2)
    for m, n, k in ((1, 96, 640), (8, 4096, 2048), (33, 250, 104), (200, 1000, 512), (1024, 2048, 512)):
        a = dev(torch.randn(m, k, generator=gen).to(torch.bfloat16))
        w = dev((torch.randn(n, k, generator=gen) / k ** 0.5).to(torch.bfloat16))
        ref = a.float() @ w.float().T
        for name, f in (("relu_squared", lambda v: torch.relu(v) ** 2), ("silu", torch.nn.functional.silu)):
            for weight in (w, gemm_tc.PackedWeight(w)):
                out = torch.empty(m, n, dtype=torch.bfloat16, device="cuda")
                gemm_tc.gemm(a, weight, out, activation=name)
                err = (out.float() - f(ref)).abs() / (1.0 + f(ref).abs())
                assert float(err.max()) <= 0.02, (m, n, k, name)
        plain_out = torch.empty(m, n, dtype=torch.bfloat16, device="cuda")
        gemm_tc.gemm(a, w, plain_out)
        assert float((plain_out.float() - ref).abs().max()) <= 0.05


def test_gated_product_with_squared_relu():
    from fastllm_py_b200.native import gemm_tc

    gen = torch.Generator().manual_seed(3)
    for m, inter, k in ((8, 4096, 512), (600, 2048, 512)):
        a = dev(torch.randn(m, k, generator=gen).to(torch.bfloat16))
        w = dev((torch.randn(2 * inter, k, generator=gen) / k ** 0.5).to(torch.bfloat16))
        out = torch.empty(m, inter, dtype=torch.bfloat16, device="cuda")
        if gemm_tc.gemm_swiglu(a, w, out, "relu_squared"):
            g, u = (a.float() @ w.float().T).split(inter, dim=1)
            ref = torch.relu(g) ** 2 * u
            assert float(((out.float() - ref).abs() / (1.0 + ref.abs())).max()) <= 0.03


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [40, 37, 512])
def test_pair_embedding_with_its_norm(dtype, width):
    """The rows of three requests (one starts, one goes on behind a kept token) normed, and fed tokens among them."""
    from fastllm_py_b200.native import ops

    gen = torch.Generator().manual_seed(4)
    vocab, buckets = 50, 17
    table, pairs = torch.randn(vocab, width, generator=gen).to(dtype), torch.randn(buckets + 1, width, generator=gen).to(dtype)
    w = 1 + 0.3 * torch.randn(width, generator=gen)
    cfg = {"embedding": {"scale": 3.0, "bigram": {"buckets": buckets, "mul_prev": 6, "mul_cur": 11}}}
    seqs = [[3, 8, 20, 41], [49, 1, 1], [7]]
    want = [plain.rms(plain.embed(cfg, {"embed": table, "bigram": pairs}, s), 1e-5) * w.double() for s in seqs]
    entries = [(0, 2, 2), (1, 0, 3), (2, 0, 1)]
    step, starts = step_of(entries, {0: 1, 1: 3, 2: 0})
    step.token_ids = i32(20, -1 - 1, 49, 1, 1, 7)
    step.token_feed, step.status = i32(9, 41), i32(0)
    last = i32(99, 8, 99, 99)
    out = torch.empty(6, width, device="cuda")
    ops.pair_embed(dev(table), dev(pairs), out, step, last, buckets, 6, 11, 3.0, dev(w), 1e-5)
    for i, (r, a, n) in enumerate(entries):
        assert float((out[starts[i]:starts[i + 1]].double().cpu() - want[r][a:a + n]).abs().max()) <= 1e-5
    assert last.tolist() == [7, 41, 99, 1] and step.status.item() == 0


@pytest.mark.parametrize("dim,vdim,heads,kv_heads", [(32, 64, 4, 2), (48, 16, 6, 2), (128, 128, 2, 1), (24, 40, 3, 3)])
def test_attention_kernels_gate_their_result(dim, vdim, heads, kv_heads):
    """A gate per channel in the CUDA-core, the tensor-core and the split-key kernel equals the kernel without it times
    the sigmoid."""
    from fastllm_py_b200.native import ops

    gen = torch.Generator().manual_seed(dim)
    page, ctx_lens, q_lens = 16, [37, 150, 0], [100, 1, 70]
    n, pages = sum(q_lens), [-(-(c + q) // page) for c, q in zip(ctx_lens, q_lens)]
    cache = dev((torch.randn(sum(pages), kv_heads, page, dim + vdim, generator=gen) * 0.7).to(torch.bfloat16))
    bt = torch.zeros(3, 16, dtype=torch.int32)
    at = 0
    for r, c in enumerate(pages):
        bt[r, :c] = torch.arange(at, at + c)
        at += c
    bt = dev(bt)
    step, starts = step_of([(r, c, q) for r, (c, q) in enumerate(zip(ctx_lens, q_lens))], {0: 0, 1: 1, 2: 2})
    q = dev((torch.randn(n, heads * dim, generator=gen) * 0.7).to(torch.bfloat16))
    wide = dev(torch.randn(n, heads * vdim + 8, generator=gen).to(torch.bfloat16))
    gate = wide[:, 8:]
    sink = torch.zeros(heads, device="cuda")
    outs = {}
    for g in (None, gate):
        simt, tc = (torch.empty(n, heads * vdim, dtype=torch.bfloat16, device="cuda") for _ in range(2))
        ops.sink_attention_simt(q, simt, cache, bt, step.tok_req, step.positions, heads, kv_heads, dim, vdim, None, 0, dim ** -0.5,
                                None, None, None, sink, page, gate=g)
        if ops.sink_tc_takes(torch.bfloat16, dim, vdim):
            ops.sink_attention_tc(q, tc, cache, bt, step, heads, kv_heads, dim, vdim, None, 0, dim ** -0.5, None, None, None, sink,
                                  page, gate=g)
        else:
            tc.copy_(simt)
        split = simt.clone()
        n_splits, kept = ops.sink_decode_splits(None, 0, 151)
        split[starts[1]] = 0
        ops.sink_decode(q, split, cache, bt, step.tok_req, step.positions, i32(starts[1]),
                        torch.empty(heads * n_splits * (vdim + 2), device="cuda"), n_splits, kept, heads, kv_heads, dim, vdim, None, 0,
                        dim ** -0.5, None, None, None, sink, page, gate=g)
        outs[g is not None] = (simt, tc, split)
    for plain_out, gated in zip(outs[False], outs[True]):
        ref = plain_out.float() * torch.sigmoid(gate.float())
        assert float((gated.float() - ref).abs().max()) <= 0.02
        assert float((gated.float() - plain_out.float()).abs().max()) > 0.1


def test_other_arrangements_of_the_parts(tmp_path):
    """The sum of two linear attentions, a convolved attention with an output bias in a block that cannot defer it (a scaled
    residual), and beside another mixer under norms: built as plans by hand, cut against cut."""
    from fastllm_py_b200 import StepEntry
    from fastllm_py_b200.api import _RandomSpec
    from fastllm_py_b200.config import EngineConfig
    from fastllm_py_b200.engine import Engine
    from fastllm_py_b200.parts import BuildContext, Decoder, LayerRun, LayerSpec, ModelPlan, PartSpec
    from fastllm_py_b200.weights import RandomStore
    from fastllm_py_b200.weights.loader import load_tensors

    W, eps = 40, 1e-5
    norm = lambda name: PartSpec("rmsnorm", dict(size=W, eps=eps), {"weight": name})

    def gla(at, heads, dim, vdim):
        return PartSpec("gated_linear_attention", dict(hidden_size=W, heads=heads, dim=dim, vdim=vdim, tau=4.0, rank=5, norm_eps=eps),
                        {s: at + s for s in ("q", "k", "v", "g", "o", "norm", "a1", "a2", "a2_bias")})

    def attention(at):
        names = ("q", "k", "v", "o", "q_bias", "k_bias", "v_bias", "o_bias", "q_conv", "k_conv", "v_conv", "q_norm", "k_norm", "gate")
        return PartSpec("normed_attention", dict(hidden_size=W, heads=4, kv_heads=2, dim=16, vdim=16, scale=0.25, norm_eps=eps,
                                                 qk_norm="weighted", biases=True, out_bias=True, taps=3, sink="unit",
                                                 channel_gate=True), {s: at + s for s in names})
    layers = [LayerSpec("prenorm", PartSpec("side_by_side_sum", dict(hidden_size=W, left=gla("a.l.", 2, 8, 12), right=gla("a.r.", 3, 4, 5),
                                                                      left_scale=0.5, right_scale=-0.7)), None, {"mixer": norm("a.n")}),
              LayerSpec("prenorm", attention("b."), None, {"mixer": norm("b.n")}, params=dict(residual_scale=0.6)),
              LayerSpec("prenorm", PartSpec("side_by_side", dict(hidden_size=W, norm_eps=eps, left=attention("c.l."),
                                                                  right=gla("c.r.", 2, 8, 8)), {"left_out": "c.lo", "right_out": "c.ro"}),
                        None, {"mixer": norm("c.n")})]
    io = dict(vocab_size=50, hidden_size=W)
    toks = np.random.default_rng(3).integers(0, 50, size=60).tolist()
    for dtype in ("float32", "bfloat16"):
        plan = ModelPlan(hidden_size=W, vocab_size=50, max_positions=64, embedding=PartSpec("table", io, {"weight": "e"}), layers=layers,
                         order=[LayerRun(0), LayerRun(1), LayerRun(2)], final_norm=norm("f"), head=PartSpec("linear", io, {"weight": "h"}))
        ctx = BuildContext(torch.device("cuda"), getattr(torch, dtype), 8, 64)
        dec = Decoder(plan, ctx)
        assert {(1, "kv"), (1, "conv"), (0, "left"), (0, "right"), (2, "left.kv"), (2, "left.conv"), (2, "right")} == set(dec.cache_needs())
        expected = dec.expected_tensors()
        dec.load(load_tensors(expected, RandomStore(expected, 3, 0.3, 0.3, torch.bfloat16), torch.device("cuda")))
        eng = Engine(dec, EngineConfig(dtype=dtype, page_size=8, max_requests=2, max_batched_tokens=64, cuda_graph=False), 64, 16)
        whole = replay.run_in_process(eng, replay.whole({"a": toks}))
        spread = float(torch.stack(list(whole.values())).std())
        assert spread > 0.05
        for steps in (replay.portions({"a": toks}, (5, 2, 9)), replay.tail_decode({"a": toks}, 50)):
            got = replay.run_in_process(eng, steps)
            err = max(float((got[k] - whole[k]).abs().max()) for k in whole)
            assert err <= (1e-5 if dtype == "float32" else 0.15) * spread, (dtype, err, spread)
        # the output bias reaches the logits, also where the block does not add it
        for part in (dec.blocks[1].mixer, dec.blocks[2].mixer.left):
            assert not part.defers_out_bias and part.out_bias is not None
            part.out_bias += 1.0
            moved = replay.run_in_process(eng, replay.whole({"a": toks}))
            assert max(float((moved[k] - whole[k]).abs().max()) for k in whole) > 0.05 * spread
            whole = moved
