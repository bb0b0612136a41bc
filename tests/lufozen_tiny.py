"""Small Lufozen configurations and weights for the tests.

`config(...)` builds the raw config.json dict from layer descriptions, `weights(raw, seed)` draws
every tensor (bfloat16, like a stored model), `write(raw, tensors, folder)` makes a model folder.
The spread of each kind of tensor is chosen so that every mechanism matters: stored norm weights
away from 0, biases and convolution taps of both signs, decays between 0.3 and 1, gates of both signs.
"""
from __future__ import annotations

import json
import sys
from pathlib import Path

import torch

ROOT = Path(__file__).resolve().parent.parent
if str(ROOT) not in sys.path:
    sys.path.insert(0, str(ROOT))


def _softmax(heads, kv_heads, dim, vdim, scale, rot, base, scaling):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale if scale is not None else dim ** -0.5, "vdim": vdim}
    if rot is not None:
        m["rot"] = {"base": base, "dims": rot}
        if scaling is not None:
            factor, original, low, high = scaling
            m["rot"]["scaling"] = {"factor": factor, "high": high, "low": low, "original": original}
    return m


def attention(heads=4, kv_heads=2, dim=16, vdim=24, conv=4, rot=8, base=10000.0, scaling=None, scale=None):
    """The lone attention: biases, convolution, interleaved pairs, one more in the denominator, a gate per channel."""
    m = _softmax(heads, kv_heads, dim, vdim, scale, rot, base, scaling)
    if conv is not None:
        m["conv"] = conv
    return {"type": "attention", "mixer": m}


def linear(heads=2, dim=8, vdim=12, tau=8.0):
    return {"type": "gla", "mixer": {"dim": dim, "heads": heads, "tau": tau, "vdim": vdim}}


def left(heads=4, kv_heads=2, dim=16, vdim=12, rot=8, base=10000.0, scaling=None, scale=None):
    return _softmax(heads, kv_heads, dim, vdim, scale, rot, base, scaling)


def right(heads=4, vdim=8, state=12, groups=2, conv=4, norm_groups=2):
    return {"conv": conv, "groups": groups, "heads": heads, "norm_groups": norm_groups, "state": state, "vdim": vdim}


def pair(l, r, left_scale=0.7, right_scale=0.4):
    return {"type": "parallel", "mixer": {"left": l, "left_scale": left_scale, "right": r, "right_scale": right_scale}}


def dense(ff=48):
    return {"ff": ff, "kind": "dense"}


def config(layers, vocab=97, width=40, eps=1e-5, loop=None, buckets=53, mul=(13, 5), scale=4.0, logit_scale=0.7):
    """`layers`: (mixer entry, mlp) pairs; loop: (start, stop, times) or None; buckets None: no table of token pairs."""
    emb = {"scale": scale}
    if buckets is not None:
        emb["bigram"] = {"buckets": buckets, "mul_cur": mul[1], "mul_prev": mul[0]}
    raw = {"architecture": "Lufozen", "embedding": emb,
           "layers": [{"mixer": m["mixer"], "mlp": f, "type": m["type"]} for m, f in layers], "logit_scale": logit_scale,
           "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop is not None:
        raw["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return raw


def _attention_shapes(out, p, m, w, lone):
    rows = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
    for s, n in rows.items():
        out[p + s] = (n, w)
        if lone:
            out[p + s + ".b"] = (n,)
            if "conv" in m:
                out[p + s + ".conv"] = (n, m["conv"])
    out[p + "o"] = (w, m["heads"] * m["vdim"])
    out[p + "q.norm"] = out[p + "k.norm"] = (m["dim"],)
    if lone:
        out[p + "o.b"], out[p + "g"] = (w,), (m["heads"] * m["vdim"], w)


def tensor_shapes(raw, rank=6) -> dict:
    """`rank`: the inner size of the gated linear attention's decay matrices (config.json does not hold it)."""
    w = raw["width"]
    out = {"embed": (raw["vocab"], w), "embed.norm": (w,), "final.norm": (w,), "head": (raw["vocab"], w)}
    if "bigram" in raw["embedding"]:
        out["bigram"] = (raw["embedding"]["bigram"]["buckets"] + 1, w)
    if "loop" in raw:
        out["loop.step"] = (raw["loop"]["times"], w)
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        mx = p + "mix."
        out[p + "norm1"] = (w,)
        if layer["type"] == "attention":
            _attention_shapes(out, mx, m, w, True)
        elif layer["type"] == "gla":
            hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            out[mx + "q"] = out[mx + "k"] = (hd, w)
            out[mx + "v"] = out[mx + "g"] = (hv, w)
            out[mx + "o"], out[mx + "norm"] = (w, hv), (m["vdim"],)
            out[mx + "a1"], out[mx + "a2"], out[mx + "a2.b"] = (rank, w), (hd, rank), (hd,)
        else:
            _attention_shapes(out, mx + "left.", m["left"], w, False)
            r, q = m["right"], mx + "right."
            inner, bc = r["heads"] * r["vdim"], 2 * r["groups"] * r["state"]
            out[q + "in"] = (2 * inner + bc + r["heads"], w)
            out[q + "conv"], out[q + "conv.b"] = (inner + bc, r["conv"]), (inner + bc,)
            out[q + "dt_bias"] = out[q + "A_log"] = out[q + "D"] = (r["heads"],)
            out[q + "norm"], out[q + "o"] = (inner,), (w, inner)
        if layer["mlp"] is not None:
            out[p + "norm2"] = (w,)
            out[p + "mlp.up"], out[p + "mlp.down"] = (layer["mlp"]["ff"], w), (w, layer["mlp"]["ff"])
    return out


def weights(raw, seed=0, gain=1.0, rank=6, slow=False) -> dict:
    """`gain` scales all matrices; `slow`: decays close to one in both recurrences, so that far tokens still count."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(raw, rank).items():
        leaf = name.split(".")[-1]

        def randn(std):
            return torch.randn(shape, generator=gen) * std

        if name.endswith(("q.norm", "k.norm")) or name.endswith(("mix.norm", "right.norm")):
            t = 1.0 + randn(0.3)
        elif leaf in ("norm1", "norm2", "norm"):             # stored around zero
            t = randn(0.3)
        elif name.endswith("a2.b"):
            t = (4.0 if slow else 1.0) + randn(1.0)          # sigmoid(z)^(1/tau): decays near one
        elif leaf == "b":
            t = randn(0.3)
        elif leaf == "conv":
            t = randn(0.6)
        elif leaf == "dt_bias":
            t = (-5.0 if slow else -1.0) + randn(0.7)        # softplus: small steps
        elif leaf == "A_log":
            t = (-1.0 if slow else 0.3) + randn(0.5)
        elif leaf == "D":
            t = 1.0 + randn(0.5)
        elif leaf == "step":
            t = randn(0.7)
        elif name in ("embed", "bigram"):
            t = randn(0.6 if name == "embed" else 1.5)
        elif leaf == "a2":
            t = randn(2.0 / shape[1] ** 0.5)
        else:
            t = randn(gain * 1.2 / shape[1] ** 0.5)
        out[name] = t.to(torch.bfloat16)
    return out


def write(raw, tensors, folder):
    from safetensors.torch import save_file

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(raw, indent=1))
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))
    return folder
