"""Small Kerirax configurations and weights for the tests.

`config(...)` builds the raw config.json dict from layer descriptions, `weights(raw, seed)` draws
every tensor (bfloat16, like a stored model), `write(raw, tensors, folder)` makes a model folder.
The spread of each kind of tensor is chosen so that every mechanism matters: norm weights away from
1, convolution taps of both signs, decays between 0.2 and 1, gates and sinks of both signs, expert
inputs beyond the clamp.
"""
from __future__ import annotations

import json
import sys
from pathlib import Path

import torch

ROOT = Path(__file__).resolve().parent.parent
if str(ROOT) not in sys.path:
    sys.path.insert(0, str(ROOT))


def latent(heads=2, dim=12, rot_dim=8, vdim=20, kv_rank=16, q_rank=24, base=10000.0, scale=None):
    return {"type": "latent_attention",
            "mixer": {"dim": dim, "heads": heads, "kv_rank": kv_rank, "q_rank": q_rank, "rot": {"base": base, "dims": rot_dim},
                      "rot_dim": rot_dim, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "vdim": vdim}}


def left(heads=4, kv_heads=2, dim=16, vdim=12, rot=8, base=10000.0, factor=2.0, scale=None):
    """rot None: no rotation; factor None: no scaling."""
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale if scale is not None else dim ** -0.5, "vdim": vdim}
    if rot is not None:
        m["rot"] = {"base": base, "dims": rot}
        if factor is not None:
            m["rot"]["scaling"] = {"factor": factor}
    return m


def right(inner=40, state=12, dt_rank=6, conv=4):
    return {"conv": conv, "dt_rank": dt_rank, "inner": inner, "state": state}


def pair(l, r, left_scale=0.7, right_scale=0.4):
    return {"type": "parallel", "mixer": {"left": l, "left_scale": left_scale, "right": r, "right_scale": right_scale}}


def dense(ff=48):
    return {"ff": ff, "kind": "dense"}


def moe(experts=6, top=2, ff=24, limit=1.5):
    return {"expert": {"ff": ff, "limit": limit}, "kind": "moe", "router": {"experts": experts, "top": top}}


def config(layers, vocab=97, width=40, eps=1e-5, loop=None, scale=2.0, cap=20.0):
    """`layers`: (mixer entry, mlp) pairs; loop: (start, stop, times) or None; cap None: no soft cap."""
    raw = {"architecture": "Kerirax", "embedding": {"scale": scale},
           "layers": [{"mixer": m["mixer"], "mlp": f, "type": m["type"]} for m, f in layers],
           "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if cap is not None:
        raw["logit_softcap"] = cap
    if loop is not None:
        raw["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return raw


def _unit(out, p, ff, w):
    out[p + "gate"] = out[p + "up"] = (ff, w)
    out[p + "down"] = (w, ff)


def tensor_shapes(raw) -> dict:
    w = raw["width"]
    out = {"embed": (raw["vocab"], w), "final.norm": (w,), "head": (raw["vocab"], w)}
    if "loop" in raw:
        out["loop.in"], out["loop.step"] = (w, 2 * w), (raw["loop"]["times"], w)
    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        mx = p + "mix."
        out[p + "norm1"] = (w,)
        if layer["type"] == "latent_attention":
            out[mx + "dq"], out[mx + "dq.norm"] = (m["q_rank"], w), (m["q_rank"],)
            out[mx + "uq"] = (m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"])
            out[mx + "dkv"], out[mx + "dkv.norm"] = (m["kv_rank"] + m["rot_dim"], w), (m["kv_rank"],)
            out[mx + "uk"], out[mx + "uv"] = (m["heads"] * m["dim"], m["kv_rank"]), (m["heads"] * m["vdim"], m["kv_rank"])
            out[mx + "sink"], out[mx + "o"] = (m["heads"],), (w, m["heads"] * m["vdim"])
        else:
            a, q = m["left"], mx + "left."
            qc, kc = a["heads"] * a["dim"], a["kv_heads"] * a["dim"]
            out[q + "q"], out[q + "k"], out[q + "v"] = (qc, w), (kc, w), (a["kv_heads"] * a["vdim"], w)
            out[q + "q.norm"], out[q + "k.norm"], out[q + "g"] = (qc,), (kc,), (a["heads"], w)
            out[q + "o"] = (w, a["heads"] * a["vdim"])
            r, q = m["right"], mx + "right."
            n = r["inner"]
            out[q + "in"], out[q + "conv"], out[q + "conv.b"] = (2 * n, w), (n, r["conv"]), (n,)
            out[q + "x"], out[q + "dt"], out[q + "dt.b"] = (r["dt_rank"] + 2 * r["state"], n), (n, r["dt_rank"]), (n,)
            out[q + "A_log"], out[q + "D"], out[q + "o"] = (n, r["state"]), (n,), (w, n)
        f = layer["mlp"]
        if f is not None and f["kind"] == "dense":
            _unit(out, p + "mlp.", f["ff"], w)
        elif f is not None:
            out[p + "mlp.router"] = (f["router"]["experts"], w)
            for e in range(f["router"]["experts"]):
                _unit(out, f"{p}mlp.e{e}.", f["expert"]["ff"], w)
    return out


def weights(raw, seed=0, gain=1.0, slow=False) -> dict:
    """`gain` scales all matrices; `slow`: decays close to one, so that far tokens still count."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(raw).items():
        leaf = name.split(".")[-1]

        def randn(std):
            return torch.randn(shape, generator=gen) * std

        if leaf in ("norm1", "norm"):
            t = 1.0 + randn(0.3)
        elif name.endswith("dt.b"):
            t = (-4.5 if slow else -1.0) + randn(0.7)        # softplus: small steps
        elif leaf == "b":
            t = randn(0.3)
        elif leaf == "conv":
            t = randn(0.6)
        elif leaf == "A_log":
            t = (-1.0 if slow else 0.0) + randn(0.6)
        elif leaf == "D":
            t = 1.0 + randn(0.5)
        elif leaf == "sink":
            t = randn(1.5)
        elif leaf == "step":
            t = randn(0.7)
        elif name == "embed":
            t = randn(0.6)
        elif leaf == "router":
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
