"""Rezelix written out slowly: one function per mechanism, whole sequences, no cache, no batch, 64-bit unless told
otherwise.  It shares nothing with the engine; the tests compare the engine with it.

A model is ``(config, tensors)``: the dict of ``config.json`` and a dict name -> tensor.

    start:   x = N(E[token])                                                      N(x) = x / sqrt(mean(x^2) + eps) * w
    layer:   x <- x + s1 * mixer(N1(x));  x <- x + s2 * ff(N2(x))                 s1, s2: a factor a column
    logits:  head . N(x)
"""

from __future__ import annotations

import math

import torch


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def yarn(rot):
    """(frequencies, amplitude) of a rotation table: pairs that turn often within the original context keep their
    frequency, pairs that turn seldom are slowed by the factor, a ramp over the pair index between."""
    dims, base, scaling = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0

    def pair_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_of(scaling["fast"])), 0)
    hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
    slowed = []
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        slowed.append(f[i] / scaling["factor"] * ramp + f[i] * (1.0 - ramp))
    return slowed, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_halves(x, positions, rot):
    """x [tokens, heads, d]: of the first `dims` columns, the pairs (i, i + dims/2) turn by position * f_i and grow by
    the amplitude; the other columns keep their values."""
    if rot is None:
        return x
    half = rot["dims"] // 2
    f, amplitude = yarn(rot)
    a = (positions.to(torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)[None, :])[:, None, :]
    cos, sin = (a.cos() * amplitude).to(x.dtype), (a.sin() * amplitude).to(x.dtype)
    u, v = x[..., :half], x[..., half : 2 * half]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half :]], dim=-1)


def softmax_of_the_past(scores):
    """scores [n, n]: softmax over j <= i."""
    n = scores.shape[0]
    later = torch.arange(n)[None, :] > torch.arange(n)[:, None]
    return torch.softmax(scores.masked_fill(later, -math.inf), dim=-1)


def cap(scores, softcap):
    return scores if softcap is None else softcap * torch.tanh(scores / softcap)


def attention(h, w, m, eps):
    """w: the mixer's tensors by their short names; m: the mixer's entry of the config.  A value is the key as projected."""
    n = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    positions = torch.arange(n)
    values = (h @ w["k"].T).view(n, G, d)
    q = unit_rms(rotate_halves((h @ w["q"].T).view(n, H, d), positions, m.get("rot")), eps)
    k = unit_rms(rotate_halves(values, positions, m.get("rot")), eps)
    out = []
    for head in range(H):
        own = head // (H // G)
        scores = cap((q[:, head] @ k[:, own].T) * m["scale"], m.get("softcap"))
        out.append(softmax_of_the_past(scores) @ values[:, own])
    return torch.cat(out, dim=-1) @ w["o"].T


def latent_attention(h, w, m, eps):
    n = h.shape[0]
    H, d, r, v, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = torch.arange(n)
    q = (h @ w["q"].T).view(n, H, d + r)
    q_plain, q_turned = q[..., :d], rotate_halves(q[..., d:], positions, m["rot"])
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    k_turned = rotate_halves(down[:, None, rank:], positions, m["rot"])[:, 0]
    keys = (c @ w["uk"].T).view(n, H, d)
    values = (c @ w["uv"].T).view(n, H, v)
    out = []
    for head in range(H):
        scores = (q_plain[:, head] @ keys[:, head].T + q_turned[:, head] @ k_turned.T) * m["scale"]
        out.append(softmax_of_the_past(scores) @ values[:, head])
    return (torch.cat(out, dim=-1) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def short_convolution(x, taps, bias):
    """y_t = b + sum_j taps[:, last - j] * x_(t - j), zeros before the start."""
    y = bias.expand_as(x).clone()
    for back in range(min(taps.shape[1], x.shape[0])):
        y[back:] += taps[:, taps.shape[1] - 1 - back] * x[: x.shape[0] - back]
    return y


def block_diagonal(u, mats, bias):
    """u [n, blocks * size] through one [out, in] matrix a block, plus its bias."""
    parts = u.view(u.shape[0], mats.shape[0], -1)
    return (torch.einsum("tbi,boi->tbo", parts, mats) + bias).reshape(u.shape)


def gated_linear_recurrence(u, r, i, lam):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a = -8 r softplus(lam), from S = 0."""
    log_a = -8.0 * r * softplus(lam)
    a = torch.exp(log_a)
    into = torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    S, out = torch.zeros_like(u[0]), []
    for t in range(u.shape[0]):
        S = a[t] * S + into[t]
        out.append(S)
    return torch.stack(out)


def rglru(h, w, m):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = short_convolution(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    r = torch.sigmoid(block_diagonal(u, w["ra"], w["ra.b"]))
    i = torch.sigmoid(block_diagonal(u, w["ri"], w["ri.b"]))
    return (gated_linear_recurrence(u, r, i, w["lam"]) * y) @ w["o"].T


def feed_forward(h, w):
    g = h @ w["gate"].T
    return (g * torch.sigmoid(g) * (h @ w["up"].T)) @ w["down"].T


def sub(tensors, prefix, dtype):
    cut = len(prefix) + 1
    return {name[cut:]: t.to(dtype) for name, t in tensors.items() if name.startswith(prefix + ".")}


def mix(kind, h, w, m, eps):
    if kind == "attention":
        return attention(h, w, m, eps)
    if kind == "latent_attention":
        return latent_attention(h, w, m, eps)
    return rglru(h, w, m)


def forward(config, tensors, tokens, dtype=torch.float64, streams=None):
    """Logits [len(tokens), vocab]; ``streams``, a list, receives the residual stream after every layer."""
    eps = config["norm"]["eps"]
    t = {name: value.to(dtype) for name, value in tensors.items()}
    x = rms_norm(t["embed"][torch.as_tensor(tokens, dtype=torch.long)], t["embed.norm"], eps)
    for index, layer in enumerate(config["layers"]):
        p = f"l{index}"
        h = rms_norm(x, t[f"{p}.norm1"], eps)
        x = x + t[f"{p}.ls1"] * mix(layer["type"], h, sub(tensors, f"{p}.mix", dtype), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            h = rms_norm(x, t[f"{p}.norm2"], eps)
            x = x + t[f"{p}.ls2"] * feed_forward(h, sub(tensors, f"{p}.mlp", dtype))
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, t["final.norm"], eps) @ t["head"].T
