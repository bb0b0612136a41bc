"""A plain, slow Kerirax: whole sequences, float64, one function per mechanism.

Nothing here is shared with the engine: it reads a raw config dict (the nested
config.json form) and a dict of tensors by checkpoint name, and walks the
tokens of ONE sequence with loops and dense matrices.  It is the oracle of
tests/test_kerirax_*.py.

Notation: h is a layer's normed input [T, width]; W x means x @ W^T.  `alter` (a set of words)
changes one reading at a time, for the tests that must tell a right engine from a nearly right one.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def embed(cfg, tensors, tokens):
    ids = torch.as_tensor(tokens, dtype=torch.long)
    return tensors["embed"].to(F)[ids] * cfg.get("embedding", {}).get("scale", 1.0)


def enter_pass(x, x0, tensors, t, alter=()):
    """What a pass of the looped layers starts with: a product of the stream beside the embedding output, then the
    pass's vector."""
    if "no_rejoin" not in alter:
        pair = [x0, x] if "swapped_rejoin" in alter else [x, x0]
        x = torch.cat(pair, dim=-1) @ tensors["loop.in"].to(F).T
    if "no_step" not in alter:
        x = x + tensors["loop.step"].to(F)[t]
    return x


def rotary_frequencies(dims, base, scaling=None):
    """f [dims / 2], each divided by the factor of a linear scaling."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F)
    return f if scaling is None else f / float(scaling["factor"])


def rotate(x, rot, first=0, pairing="interleaved"):
    """x [T, heads, d]: the first rot["dims"] dimensions of every head turn by the position's angles, in pairs
    (2i, 2i + 1)."""
    dims = rot["dims"]
    f = rotary_frequencies(dims, rot["base"], rot.get("scaling"))
    ang = torch.arange(first, first + x.shape[0], dtype=F)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    out = x.clone()
    a = slice(0, dims, 2) if pairing == "interleaved" else slice(0, dims // 2)
    b = slice(1, dims, 2) if pairing == "interleaved" else slice(dims // 2, dims)
    u, v = x[..., a], x[..., b]
    out[..., a] = u * c - v * s
    out[..., b] = v * c + u * s
    return out


def softmax_attention(q, k, v, scale, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv], causal; `sink` [H]: exp(sink) more in the denominator."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F)
    hidden = torch.triu(torch.ones(T, T, dtype=torch.bool), 1)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * scale
        s = s.masked_fill(hidden, -math.inf)
        top = s.max(dim=1, keepdim=True).values
        if sink is not None:
            top = torch.clamp(top, min=float(sink[hd]))
        e = torch.exp(s - top)
        den = e.sum(1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[hd] - top)
        out[:, hd] = (e / den) @ v[:, g]
    return out


def latent_attention(h, t, m, eps, alter=()):
    """Queries through a normed latent, keys and values from a normed latent, one rotated key part for all heads, a
    sink in the denominator."""
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pairing = "half" if "other_pairing" in alter else "interleaved"
    cq = h @ t["dq"].T
    if "no_query_norm" not in alter:
        cq = rms(cq, eps) * t["dq.norm"]
    q = (cq @ t["uq"].T).view(T, H, d + r)
    q = torch.cat([q[..., :d], rotate(q[..., d:], m["rot"], pairing=pairing)], dim=-1)
    kv = h @ t["dkv"].T
    c = rms(kv[:, :rank], eps) * t["dkv.norm"]
    shared = rotate(kv[:, None, rank:], m["rot"], pairing=pairing)
    k = torch.cat([(c @ t["uk"].T).view(T, H, d), shared.expand(T, H, r)], dim=-1)
    v = (c @ t["uv"].T).view(T, H, dv)
    o = softmax_attention(q, k, v, m["scale"], None if "no_sink" in alter else t["sink"])
    return o.reshape(T, H * dv) @ t["o"].T


def left_attention(h, t, m, eps, alter=()):
    """Queries and keys normed over their whole projections, rotated pairs, an ordinary softmax, a gate per head."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = h @ t["q"].T, h @ t["k"].T
    if "head_norm" in alter:
        q, k = rms(q.view(T, H, d), eps).reshape(T, -1), rms(k.view(T, G, d), eps).reshape(T, -1)
    else:
        q, k = rms(q, eps), rms(k, eps)
    q, k = (q * t["q.norm"]).view(T, H, d), (k * t["k.norm"]).view(T, G, d)
    if m.get("rot") is not None:
        rot = dict(m["rot"], scaling=None) if "no_scaling" in alter else m["rot"]
        pairing = "half" if "other_pairing" in alter else "interleaved"
        q, k = rotate(q, rot, pairing=pairing), rotate(k, rot, pairing=pairing)
    o = softmax_attention(q, k, (h @ t["v"].T).view(T, G, dv), m["scale"])
    if "no_gate" not in alter:
        o = o * torch.sigmoid(h @ t["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ t["o"].T


def short_conv(u, w, bias, tail):
    """y_t = sum_j w[:, j] u_(t - taps + 1 + j) + bias: u [T, channels], w [channels, taps]; `tail`: the taps - 1 rows
    before u."""
    taps, T = w.shape[1], u.shape[0]
    us = torch.cat([tail, u], dim=0)
    y = sum(us[j:j + T] * w[:, j] for j in range(taps))
    return y + bias


def selective_scan(h, t, m, state=None, alter=()):
    """A recurrence per channel and state element whose step size, input and read-out vectors are made from the token.
    state: None or (S [inner, state], the last taps - 1 inputs of the convolution); returns (output, new state)."""
    T = h.shape[0]
    inner, N, rank, taps = m["inner"], m["state"], m["dt_rank"], m["conv"]
    proj = h @ t["in"].T
    u, z = proj[:, :inner], proj[:, inner:]
    S, tail = (torch.zeros(inner, N, dtype=F), torch.zeros(taps - 1, inner, dtype=F)) if state is None else state
    x = silu(short_conv(u, t["conv"], t["conv.b"], tail))
    new_tail = torch.cat([tail, u], dim=0)[T:]
    low = x @ t["x"].T
    dt = low[:, :rank] @ t["dt"].T + (0.0 if "no_dt_bias" in alter else t["dt.b"])
    dt = torch.nn.functional.softplus(dt)
    B, C = low[:, rank:rank + N], low[:, rank + N:]
    A = -torch.exp(t["A_log"])
    y = torch.zeros(T, inner, dtype=F)
    for i in range(T):
        S = torch.exp(dt[i][:, None] * A) * S + (dt[i] * x[i])[:, None] * B[i][None, :]
        y[i] = S @ C[i]
    if "no_skip" not in alter:
        y = y + t["D"] * x
    return (y * silu(z)) @ t["o"].T, (S, new_tail)


def pair(h, t, m, eps, alter=()):
    left = left_attention(h, sub(t, "left."), m["left"], eps, alter)
    right, _ = selective_scan(h, sub(t, "right."), m["right"], alter=alter)
    ls, rs = m.get("left_scale", 1.0), m.get("right_scale", 1.0)
    if "swapped_scales" in alter:
        ls, rs = rs, ls
    return ls * left + rs * right


def gated_unit(h, t):
    return (silu(h @ t["gate"].T) * (h @ t["up"].T)) @ t["down"].T


def clamped_expert(h, t, limit):
    g = torch.clamp(h @ t["gate"].T, max=limit)
    u = torch.clamp(h @ t["up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ t["down"].T


def routed_experts(h, t, m, alter=()):
    """Every token's `top` experts by sigmoid score; the score multiplies what the expert reads."""
    top, limit = m["router"]["top"], m["expert"]["limit"]
    s = torch.sigmoid(h @ t["router"].T)
    y = torch.zeros_like(h)
    for i in range(h.shape[0]):
        for e in torch.argsort(-s[i], stable=True)[:top].tolist():
            te = sub(t, f"e{e}.")
            w = s[i, e] / s[i].topk(top).values.sum() if "renormalised" in alter else s[i, e]
            if "weight_on_output" in alter:
                y[i] += w * clamped_expert(h[i], te, limit)
            else:
                y[i] += clamped_expert(w * h[i], te, limit)
    return y


def sub(tensors, prefix):
    return {k[len(prefix):]: v.to(F) for k, v in tensors.items() if k.startswith(prefix)}


def mixer(kind, h, t, m, eps, alter=()):
    if kind == "parallel":
        return pair(h, t, m, eps, alter)
    if kind == "latent_attention":
        return latent_attention(h, t, m, eps, alter)
    raise ValueError(kind)


def feed_forward(h, t, m, alter=()):
    return gated_unit(h, t) if m["kind"] == "dense" else routed_experts(h, t, m, alter)


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
    x = x0 = embed(cfg, tensors, tokens)
    for i, p in running_order(cfg):
        layer = cfg["layers"][i]
        t = sub(tensors, f"l{i}.")
        if p is not None:
            x = enter_pass(x, x0, tensors, p, alter)
        h = rms(x, eps) * t["norm1"]
        y = mixer(layer["type"], h, sub(t, "mix."), layer["mixer"], eps, alter)
        if layer.get("mlp") is not None:
            if "one_after_the_other" in alter:
                x, y, h = x + y, 0.0, rms(x + y, eps) * t["norm1"]
            y = y + feed_forward(h, sub(t, "mlp."), layer["mlp"], alter)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = (rms(x, eps) * tensors["final.norm"].to(F)) @ tensors["head"].to(F).T
    cap = cfg.get("logit_softcap")
    return logits if cap is None or "no_cap" in alter else cap * torch.tanh(logits / cap)
