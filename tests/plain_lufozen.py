"""A plain, slow Lufozen: whole sequences, float64, one function per mechanism.

Nothing here is shared with the engine: it reads a raw config dict (the nested
config.json form) and a dict of tensors by checkpoint name, and walks the
tokens of ONE sequence with loops and dense matrices.  It is the oracle of
tests/test_lufozen_*.py.

Notation: h is a layer's normed input [T, width]; W x means x @ W^T.  `alter` (a set of words)
changes one reading at a time, for the tests that must tell a right engine from a nearly right one.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def model_norm(x, w, eps, alter=()):
    """An RMS norm whose stored weight is the distance from one."""
    return rms(x, eps) * (w if "plain_weight" in alter else 1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def embed(cfg, tensors, tokens, alter=()):
    """Token rows times a scale plus rows of the hashed pair table; the sequence's first token takes the last row."""
    ids = torch.as_tensor(tokens, dtype=torch.long)
    e = cfg.get("embedding", {})
    x = tensors["embed"].to(F)[ids] * e.get("scale", 1.0)
    b = e.get("bigram")
    if b is not None and "no_pairs" not in alter:
        table = tensors["bigram"].to(F)
        for i in range(len(ids)):
            row = b["buckets"]
            if i > 0:
                row = (int(ids[i - 1]) * b["mul_prev"] + int(ids[i]) * b["mul_cur"]) % b["buckets"]
            x[i] = x[i] + table[row]
    return x


def rotary_frequencies(dims, base, scaling=None):
    """f [dims / 2]; with scaling, by wavelength l = 2 pi / f against `original`: kept below original / high, divided
    by `factor` above original / low, blended between."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            factor, orig, low, high = (float(scaling[k]) for k in ("factor", "original", "low", "high"))
            wave = 2 * math.pi / f
            if wave > orig / low:
                f = f / factor
            elif wave >= orig / high:
                s = (orig / wave - low) / (high - low)
                f = (1 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=F)


def rotate(x, rot, pairing):
    """x [T, heads, d]: the first rot["dims"] dimensions of every head turn by the position's angles;
    pairing "interleaved": (2i, 2i + 1); "half": (i, i + dims / 2)."""
    dims = rot["dims"]
    f = rotary_frequencies(dims, rot["base"], rot.get("scaling"))
    out = x.clone()
    for t in range(x.shape[0]):
        for i in range(dims // 2):
            a, b = (2 * i, 2 * i + 1) if pairing == "interleaved" else (i, i + dims // 2)
            c, s = math.cos(t * float(f[i])), math.sin(t * float(f[i]))
            u, v = x[t, :, a], x[t, :, b]
            out[t, :, a] = u * c - v * s
            out[t, :, b] = v * c + u * s
    return out


def softmax_attention(q, k, v, scale, plus_one):
    """q [T, H, d], k [T, G, d], v [T, G, dv], causal; `plus_one`: one more unit in the softmax's denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    for hd in range(H):
        g = hd // (H // G)
        for i in range(T):
            s = (k[:i + 1, g] @ q[i, hd]) * scale
            top = s.max()
            if plus_one:
                top = torch.clamp(top, min=0.0)
            e = torch.exp(s - top)
            den = e.sum() + (torch.exp(-top) if plus_one else 0.0)
            out[i, hd] = (e[:, None] * v[:i + 1, g]).sum(0) / den
    return out


def short_conv(u, w, tail=None, bias=None):
    """y_t = sum_j w[:, j] u_(t - taps + 1 + j) (+ bias): u [T, channels], w [channels, taps]; `tail`: the taps - 1
    rows before u (zeros at a sequence's start)."""
    taps = w.shape[1]
    if tail is None:
        tail = torch.zeros(taps - 1, u.shape[1], dtype=F)
    us = torch.cat([tail, u], dim=0)
    y = torch.stack([(us[i:i + taps] * w.T).sum(0) for i in range(u.shape[0])])
    return y if bias is None else y + bias


def gated_attention(h, t, m, eps, alter=()):
    """Biased projections, a short convolution on q, k and v, weighted head norms, interleaved rotary pairs, a softmax
    with one added to its denominator, a gate per channel, a biased output product."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ t[s].T + t[s + ".b"] for s in ("q", "k", "v"))
    if "q.conv" in t and "no_conv" not in alter:
        q, k, v = short_conv(q, t["q.conv"]), short_conv(k, t["k.conv"]), short_conv(v, t["v.conv"])
    q = rms(q.view(T, H, d), eps) * t["q.norm"]
    k = rms(k.view(T, G, d), eps) * t["k.norm"]
    if m.get("rot") is not None:
        pairing = "half" if "other_pairing" in alter else "interleaved"
        q, k = rotate(q, m["rot"], pairing), rotate(k, m["rot"], pairing)
    o = softmax_attention(q, k, v.view(T, G, dv), m["scale"], "no_sink" not in alter).reshape(T, H * dv)
    if "no_gate" not in alter:
        o = o * torch.sigmoid(h @ t["g"].T)
    return o @ t["o"].T + (0.0 if "no_out_bias" in alter else t["o.b"])


def left_attention(h, t, m, eps, alter=()):
    """The attention of the pair: weighted head norms, rotate-half pairs, an ordinary softmax, no biases."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ t["q"].T).view(T, H, d), eps) * t["q.norm"]
    k = rms((h @ t["k"].T).view(T, G, d), eps) * t["k.norm"]
    if m.get("rot") is not None:
        pairing = "interleaved" if "other_pairing" in alter else "half"
        q, k = rotate(q, m["rot"], pairing), rotate(k, m["rot"], pairing)
    o = softmax_attention(q, k, (h @ t["v"].T).view(T, G, dv), m["scale"], "left_sink" in alter)
    return o.reshape(T, H * dv) @ t["o"].T


def state_space(h, t, m, eps, state=None, alter=()):
    """The state-space recurrence with a scalar decay per head.  state: None or (S [heads, N, vdim], the last taps - 1
    inputs of the convolution); returns (output, new state)."""
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    proj = h @ t["in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    taps = m["conv"]
    S, tail = (torch.zeros(H, N, P, dtype=F), torch.zeros(taps - 1, xbc.shape[1], dtype=F)) if state is None else state
    c = silu(short_conv(xbc, t["conv"], tail, t["conv.b"]))
    new_tail = torch.cat([tail, xbc], dim=0)[T:]
    x = c[:, :inner].view(T, H, P)
    B = c[:, inner:inner + G * N].view(T, G, N)
    C = c[:, inner + G * N:].view(T, G, N)
    dt = torch.nn.functional.softplus(dt + t["dt_bias"])
    y = torch.zeros(T, H, P, dtype=F)
    for i in range(T):
        for hd in range(H):
            g = hd // (H // G)
            decay = torch.exp(-torch.exp(t["A_log"][hd]) * dt[i, hd])
            S[hd] = decay * S[hd] + dt[i, hd] * B[i, g][:, None] * x[i, hd][None, :]
            y[i, hd] = S[hd].T @ C[i, g] + (0.0 if "no_skip" in alter else t["D"][hd] * x[i, hd])
    y = y.reshape(T, inner)
    parts = 1 if "one_norm" in alter else m["norm_groups"]
    if "norm_first" in alter:
        y = rms(y.view(T, parts, -1), eps).reshape(T, inner) * silu(z)
    else:
        y = rms((y * silu(z)).view(T, parts, -1), eps).reshape(T, inner)
    return (y * t["norm"]) @ t["o"].T, (S, new_tail)


def gated_linear_attention(h, t, m, eps, state=None, alter=()):
    """A matrix state per head whose rows (one per key channel) decay by a number made from the token.
    state: None or S [heads, dim, vdim]; returns (output, S)."""
    T = h.shape[0]
    H, d, dv, tau = m["heads"], m["dim"], m["vdim"], m["tau"]
    q = (h @ t["q"].T).view(T, H, d) * d ** -0.5
    k = (h @ t["k"].T).view(T, H, d)
    v = (h @ t["v"].T).view(T, H, dv)
    z = (h @ t["a1"].T) @ t["a2"].T + t["a2.b"]
    alpha = torch.exp(torch.nn.functional.logsigmoid(z) / tau).view(T, H, d)
    if "no_decay" in alter:
        alpha = torch.ones_like(alpha)
    S = torch.zeros(H, d, dv, dtype=F) if state is None else state
    o = torch.zeros(T, H, dv, dtype=F)
    for i in range(T):
        S = alpha[i][:, :, None] * S + k[i][:, :, None] * v[i][:, None, :]
        o[i] = torch.einsum("hdv,hd->hv", S, q[i])
    o = rms(o, eps) * t["norm"]
    return (o.reshape(T, H * dv) * silu(h @ t["g"].T)) @ t["o"].T, S


def squared_relu_unit(h, t):
    return torch.relu(h @ t["up"].T) ** 2 @ t["down"].T


def sub(tensors, prefix):
    return {k[len(prefix):]: v.to(F) for k, v in tensors.items() if k.startswith(prefix)}


def mixer(kind, h, t, m, eps, alter=()):
    if kind == "parallel":
        left = left_attention(h, sub(t, "left."), m["left"], eps, alter)
        right, _ = state_space(h, sub(t, "right."), m["right"], eps, alter=alter)
        ls, rs = m["left_scale"], m["right_scale"]
        if "swapped_scales" in alter:
            ls, rs = rs, ls
        return ls * left + rs * right
    if kind == "gla":
        return gated_linear_attention(h, t, m, eps, alter=alter)[0]
    if kind == "attention":
        return gated_attention(h, t, m, eps, alter)
    raise ValueError(kind)


def running_order(cfg):
    """[(layer, pass number or None at the first layer of a pass)]."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if loop is None:
        return [(i, None) for i in range(n)]
    start, stop = loop["start"], loop["stop"]
    out = [(i, None) for i in range(start)]
    for p in range(loop["times"]):
        out += [(i, p if i == start else None) for i in range(start, stop)]
    return out + [(i, None) for i in range(stop, n)]


def forward(cfg, tensors, tokens, layers_out=None, alter=()):
    """Logits [T, vocab] of one whole sequence.  `layers_out`: a list that receives the residual stream after
    every layer run."""
    eps = cfg["norm"]["eps"]
    x = model_norm(embed(cfg, tensors, tokens, alter), tensors["embed.norm"].to(F), eps, alter)
    for i, step in running_order(cfg):
        layer = cfg["layers"][i]
        t = sub(tensors, f"l{i}.")
        if step is not None and "no_step" not in alter:
            x = x + tensors["loop.step"].to(F)[step]
        x = x + mixer(layer["type"], model_norm(x, t["norm1"], eps, alter), sub(t, "mix."), layer["mixer"], eps, alter)
        if layer.get("mlp") is not None:
            x = x + squared_relu_unit(model_norm(x, t["norm2"], eps, alter), sub(t, "mlp."))
        if layers_out is not None:
            layers_out.append(x.clone())
    x = model_norm(x, tensors["final.norm"].to(F), eps, alter)
    return x @ tensors["head"].to(F).T * cfg.get("logit_scale", 1.0)
