"""Koravik written out slowly: one function per mechanism, whole sequences, no cache, no batch, 64-bit unless told
otherwise.  It shares nothing with the engine; the tests compare the engine with it.

A model is ``(config, tensors)``: the dict of ``config.json`` and a dict name -> tensor.

    start:   x0 = N(E[token]);  x = x0                                            N(x) = x / sqrt(mean(x^2) + eps) * w
    pass:    x <- W_in [x; x0], once, right before the first layer of every pass of the loop
    layer:   h = N1(x);  x <- x + m * sigmoid(R1 h + b1) * attention(h)
             h = N2(x);  x <- x + m * sigmoid(R2 h + b2) * ff(h)
    logits:  E . N(x) * logit_scale
"""

from __future__ import annotations

import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotate_halves(x, positions, dims, base):
    """x [tokens, heads, d]: of the first `dims` columns, the pairs (i, i + dims/2) turn by position * base^(-2i/dims)."""
    half = dims // 2
    rate = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = (positions.to(torch.float64)[:, None] * rate[None, :])[:, None, :]
    cos, sin = a.cos().to(x.dtype), a.sin().to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def visible(n, size, keep_first):
    """[n, n] bool: position i sees j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def window_of(m, n):
    """(size, kept first tokens) of a mixer's mask; without one every key stays in sight."""
    mask = m.get("mask")
    return (mask["size"], mask.get("keep_first", 0)) if mask else (n, 0)


def mix_heads(scores, talk):
    """scores [heads, n, n] -> sum over g of talk[h, g] * scores[g]."""
    return torch.einsum("hg,gij->hij", talk, scores)


def attention(h, w, m):
    """w: the mixer's tensors by their short names; m: the mixer's entry of the config."""
    n = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    positions = torch.arange(n)
    q = rotate_halves((h @ w["q"].T).view(n, H, d), positions, m["rot"]["dims"], m["rot"]["base"])
    values = (h @ w["k"].T).view(n, G, d)  # a value is the key before its turn
    k = rotate_halves(values, positions, m["rot"]["dims"], m["rot"]["base"])
    own = [head // (H // G) for head in range(H)]
    scores = torch.stack([q[:, head] @ k[:, own[head]].T for head in range(H)]) * m["scale"]
    scores = mix_heads(scores, w["talk"])
    scores = scores.masked_fill(~visible(n, *window_of(m, n)), -math.inf)
    p = torch.softmax(scores, dim=-1)
    mixed = torch.cat([p[head] @ values[:, own[head]] for head in range(H)], dim=-1)
    return mixed @ w["o"].T


def relu2_unit(h, up, down):
    return (torch.relu(h @ up.T) ** 2) @ down.T


def expert_mixture(h, w, f):
    """Every token: its `top` experts by sigmoid score (ties to the lower index), weighted by their share of the chosen
    scores' sum; the shared expert, if there is one, on top."""
    scores = torch.sigmoid(h @ w["router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = sorted(range(scores.shape[1]), key=lambda e: (-float(scores[t, e]), e))[: f["router"]["top"]]
        total = sum(scores[t, e] for e in chosen) + 1e-20
        for e in chosen:
            out[t] += scores[t, e] / total * relu2_unit(h[t], w[f"e{e}.up"], w[f"e{e}.down"])
    if f.get("shared"):
        out = out + relu2_unit(h, w["shared.up"], w["shared.down"])
    return out


def gated_sum(x, h, y, gate, bias, m):
    """The stream plus a sub-layer's result, gated element by element by what the sub-layer read."""
    return x + m * torch.sigmoid(h @ gate.T + bias) * y


def pass_input(x, x0, w_in):
    return torch.cat([x, x0], dim=-1) @ w_in.T


def sub(tensors, prefix, dtype):
    cut = len(prefix) + 1
    return {name[cut:]: t.to(dtype) for name, t in tensors.items() if name.startswith(prefix + ".")}


def run_order(config):
    """(layer index, whether a pass of the loop begins with it) in the order the layers run."""
    count = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(count)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    once = [(i, i == start) for i in range(start, stop)]
    return [(i, False) for i in range(start)] + once * times + [(i, False) for i in range(stop, count)]


def forward(config, tensors, tokens, dtype=torch.float64, streams=None):
    """Logits [len(tokens), vocab]; ``streams``, a list, receives the residual stream after every layer run."""
    eps, m = config["norm"]["eps"], config["residual_mult"]
    t = {name: value.to(dtype) for name, value in tensors.items()}
    x0 = rms_norm(t["embed"][torch.as_tensor(tokens, dtype=torch.long)], t["embed.norm"], eps)
    x = x0
    for index, begins_pass in run_order(config):
        p, layer = f"l{index}", config["layers"][index]
        if begins_pass:
            x = pass_input(x, x0, t["loop.in"])
        h = rms_norm(x, t[f"{p}.norm1"], eps)
        x = gated_sum(x, h, attention(h, sub(tensors, f"{p}.mix", dtype), layer["mixer"]), t[f"{p}.rg1"], t[f"{p}.rg1.b"], m)
        if layer.get("mlp") is not None:
            h = rms_norm(x, t[f"{p}.norm2"], eps)
            x = gated_sum(x, h, expert_mixture(h, sub(tensors, f"{p}.mlp", dtype), layer["mlp"]), t[f"{p}.rg2"], t[f"{p}.rg2.b"], m)
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, t["final.norm"], eps) @ t["embed"].T * config["logit_scale"]
