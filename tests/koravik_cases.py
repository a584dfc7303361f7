"""Small Koravik configurations and weights for the tests.

The weights are drawn so that a fault shows: queries and keys are large enough for the softmax to pick single keys (a wrong
rotation, a key just outside the window, a lost first token or a wrong key/value head then moves the result by far more than
rounding), the heads' scores are mixed strongly (every head takes a good part of its neighbours' scores, with both signs), the
residual gates are neither open nor shut, the norm weights differ from one, the routers spread their logits and a looped
layer's input takes as much of the embedding output as of the stream.  The configurations differ in every size: heads and
key/value heads (one, several, as many as heads, more than sixteen), head widths (multiples of 16 and of nothing), rotated
parts of a head and none, windows from one token up and none, kept first tokens from none to more than a page and more than
the window, one expert a token and several and all of them, mixtures with and without a shared expert, layers without a
feed-forward, loops at the start, in the middle, of one layer, of one pass, and none, other residual and logit factors.
"""

from __future__ import annotations

import json
from pathlib import Path
from typing import Any, Mapping

import torch
from safetensors.torch import save_file


def attention(heads, kv_heads, dim, scale, *, rot=None, window=None, keep=0, base=10000.0):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "rot": {"base": base, "dims": rot or dim}}
    if window is not None:
        mixer["mask"] = {"size": window, "keep_first": keep}
    return mixer


def moe(experts, top, ff, shared=None):
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


def layer(mixer, mlp):
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def config(width, vocab, layers, loop=None, eps=1e-5, residual_mult=0.7, logit_scale=1.5):
    cfg = {"architecture": "Koravik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": residual_mult, "logit_scale": logit_scale,
           "layers": layers}
    if loop is not None:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


# name -> (config, seed, page size)
CASES: dict[str, tuple[dict, int, int]] = {
    # heads of 16 and 32: the tensor-core kernels in bfloat16 (rows of no whole band: copies a lane at a time); a loop in the middle
    "looped": (config(48, 97, [
        layer(attention(6, 2, 16, 0.2, window=13, keep=3, base=500.0), moe(6, 2, 24, shared=16)),
        layer(attention(3, 1, 32, 0.25, rot=8, window=21, keep=1), moe(4, 3, 16)),
        layer(attention(2, 2, 16, 0.3, rot=4, window=34), None),
        layer(attention(4, 4, 16, 0.2, window=7, keep=9, base=300.0), moe(5, 1, 24, shared=40)),
    ], loop=(1, 3, 2)), 51, 8),
    # nothing a multiple of 8: the 32-bit-arithmetic kernel in both modes; every expert chosen; one layer that loops from the start
    "odd": (config(50, 77, [
        layer(attention(3, 3, 10, 0.4, rot=6, window=9, keep=5, base=100.0), moe(3, 3, 18, shared=10)),
        layer(attention(6, 2, 14, 0.35, rot=2, window=40, keep=17), moe(4, 2, 30)),
        layer(attention(2, 1, 6, 0.5, base=50.0), None),
    ], loop=(0, 1, 3), eps=1e-6, residual_mult=0.45, logit_scale=0.3), 52, 16),
    # no loop; key rows of whole bands (copies by TMA) and the widest; one expert of one; more than sixteen heads
    "wide": (config(64, 131, [
        layer(attention(8, 4, 64, 0.12, rot=32, window=45, keep=18, base=40000.0), moe(1, 1, 32)),
        layer(attention(20, 4, 128, 0.09, window=70, keep=2), moe(7, 2, 24, shared=40)),
        layer(attention(5, 1, 128, 0.1, rot=64), moe(3, 1, 16)),
    ], residual_mult=1.0, logit_scale=1.0), 53, 16),
    # pages of four; a loop of one pass over the end; a window of one token and a few kept ones; one head
    "small_pages": (config(32, 61, [
        layer(attention(1, 1, 16, 0.35, window=1, keep=6), moe(2, 1, 24)),
        layer(attention(10, 5, 16, 0.25, rot=8, window=18, keep=4), moe(4, 4, 8, shared=8)),
    ], loop=(1, 2, 1)), 54, 4),
}


def _normal(generator, shape, std):
    return torch.randn(shape, generator=generator, dtype=torch.float32) * std


def make_weights(cfg: Mapping[str, Any], seed: int) -> dict[str, torch.Tensor]:
    """fp32 tensors whose values are exact in bfloat16 (a model folder written in either dtype holds the same numbers)."""
    g = torch.Generator().manual_seed(seed)
    width, vocab = cfg["width"], cfg["vocab"]
    w: dict[str, torch.Tensor] = {
        "embed": _normal(g, (vocab, width), width ** -0.5), "embed.norm": 1.0 + _normal(g, (width,), 0.2), "final.norm": 1.0 + _normal(g, (width,), 0.2),
    }
    if cfg.get("loop"):
        w["loop.in"] = _normal(g, (width, 2 * width), (2 * width) ** -0.5)
    for index, entry in enumerate(cfg["layers"]):
        p, m = f"l{index}", entry["mixer"]
        heads, kv_heads, dim = m["heads"], m["kv_heads"], m["dim"]
        gain = (2.5 / (m["scale"] * dim ** 0.5)) ** 0.5  # scores of a few units: the softmax picks single keys
        w[f"{p}.norm1"] = 1.0 + _normal(g, (width,), 0.2)
        w[f"{p}.mix.q"] = _normal(g, (heads * dim, width), gain * width ** -0.5)
        w[f"{p}.mix.k"] = _normal(g, (kv_heads * dim, width), gain * width ** -0.5)
        w[f"{p}.mix.talk"] = torch.eye(heads) + _normal(g, (heads, heads), 0.6 * heads ** -0.5)
        w[f"{p}.mix.o"] = _normal(g, (width, heads * dim), (heads * dim) ** -0.5 / gain)
        w[f"{p}.rg1"] = _normal(g, (width, width), 1.5 * width ** -0.5)
        w[f"{p}.rg1.b"] = _normal(g, (width,), 0.7)
        f = entry["mlp"]
        if f is None:
            continue
        w[f"{p}.norm2"] = 1.0 + _normal(g, (width,), 0.2)
        w[f"{p}.rg2"] = _normal(g, (width, width), 1.5 * width ** -0.5)
        w[f"{p}.rg2.b"] = _normal(g, (width,), 0.7)
        ff = f["expert"]["ff"]
        for e in range(f["router"]["experts"]):
            w[f"{p}.mlp.e{e}.up"] = _normal(g, (ff, width), 1.2 * width ** -0.5)
            w[f"{p}.mlp.e{e}.down"] = _normal(g, (width, ff), ff ** -0.5)
        w[f"{p}.mlp.router"] = _normal(g, (f["router"]["experts"], width), 1.5 * width ** -0.5)
        if f.get("shared"):
            sff = f["shared"]["ff"]
            w[f"{p}.mlp.shared.up"] = _normal(g, (sff, width), 1.2 * width ** -0.5)
            w[f"{p}.mlp.shared.down"] = _normal(g, (width, sff), sff ** -0.5)
    return {name: t.to(torch.bfloat16).to(torch.float32) for name, t in w.items()}


def write_model(cfg: Mapping[str, Any], weights: Mapping[str, torch.Tensor], folder: Path, dtype: torch.dtype = torch.bfloat16) -> Path:
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    save_file({name: t.to(dtype).contiguous() for name, t in weights.items()}, str(folder / "model.safetensors"))
    return folder


def relative_error(got, want) -> float:
    """Largest over the rows of rms(difference, its mean taken off) / rms(wanted row, its mean taken off)."""
    import numpy as np

    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    ref = want - want.mean(-1, keepdims=True)
    return float((np.sqrt((d * d).mean(-1)) / np.sqrt((ref * ref).mean(-1) + 1e-30)).max())
