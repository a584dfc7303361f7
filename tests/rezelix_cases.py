"""Small Rezelix configurations and weights for the tests.

The weights are drawn so that a fault shows: scores of a few units (the softmax picks single keys: a wrong rotation, a lost
key or a wrong key/value head moves the result by far more than rounding), caps of the size of the scores, norm weights and
column factors away from one, decays from nearly 0 to nearly 1 and different from channel to channel, gates neither open nor
shut, convolutions whose every tap matters.  The configurations differ in every size, also in those a model may happen to make
equal or 1: query and key/value heads (one, some, all), rotated parts of a head and all of it and none, caps that the kernels
take by their polynomial and by the exponential, and none, latent rows that are and are not multiples of 16, values wider and
narrower than keys, one and several parts of the recurrent unit, 1 to 5 taps, units wider and narrower than the model, layers
with and without feed-forward, rotation tables of different lengths and factors, and unscaled ones.
"""

from __future__ import annotations

import json
from pathlib import Path
from typing import Any, Mapping, Optional

import torch
from safetensors.torch import save_file


def rot(dims, base=10000.0, scaling=None):
    """scaling: (factor, original, fast, slow)"""
    table = {"base": base, "dims": dims}
    if scaling is not None:
        table["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return table


def attention(heads, kv_heads, dim, scale, rot_table, softcap=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if rot_table is not None:
        mixer["rot"] = rot_table
    if softcap is not None:
        mixer["softcap"] = softcap
    return {"type": "attention", "mixer": mixer}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, scaling=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                                  "rot": rot(rot_dim, base, scaling)}}


def rglru(width, blocks, conv):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def layer(mixer, ff: Optional[int]):
    return dict(mixer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Rezelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


YARN = (5.0, 64, 8.0, 0.5)  # within 64 positions: pairs that turn eight times and more stay, half a turn and less are slowed

# name -> (config, seed, page size)
CASES: dict[str, tuple[dict, int, int]] = {
    # heads of 32 and 16, latent rows of 32: the tensor-core kernels in bfloat16; every kind of layer with and without feed-forward
    "mixed": (config(48, 97, [
        layer(rglru(64, 4, 4), 40),
        layer(attention(4, 2, 32, 0.45, rot(16, 500.0, YARN), softcap=5.0), 24),
        layer(latent(3, 16, 8, 12, 24, 0.5, 300.0, (3.0, 48, 6.0, 1.0)), None),
        layer(rglru(48, 1, 2), None),
        layer(attention(2, 2, 16, 0.6, rot(16, 50.0), softcap=30.0), None),
        layer(latent(6, 12, 4, 16, 28, 0.6, 100.0), 32),
    ]), 61, 8),
    # nothing a multiple of 8: the 32-bit-arithmetic attention in both modes, the recurrent unit by its padded parts
    "odd": (config(50, 77, [
        layer(latent(3, 6, 2, 10, 15, 0.8, 50.0, (2.0, 32, 4.0, 0.25)), 30),
        layer(rglru(42, 2, 3), None),
        layer(attention(3, 1, 10, 0.7, rot(6, 100.0, (7.0, 100, 20.0, 2.0)), softcap=3.0), 18),
        layer(rglru(27, 3, 1), 22),
        layer(attention(6, 3, 14, 0.6, None), None),
    ], eps=1e-6), 62, 16),
    # heads of 128 and 64, latent rows of 64 and 192: the tcgen05 and TMA-fed kernels in bfloat16; parts of several bands; five taps
    "wide": (config(64, 131, [
        layer(attention(4, 1, 128, 0.22, rot(128, 40000.0, (16.0, 256, 32.0, 1.0)), softcap=70.0), 96),
        layer(rglru(288, 2, 5), 64),
        layer(latent(2, 48, 16, 40, 48, 0.3, 20000.0, (4.0, 128, 16.0, 1.0)), 48),
        layer(attention(2, 2, 64, 0.3, rot(32, 300.0), softcap=12.0), None),
        layer(latent(17, 16, 32, 8, 160, 0.35), 80),
        layer(rglru(80, 1, 4), None),
    ]), 63, 16),
    # pages of four; one query head a key/value head and one key/value head for all; the narrowest rotations
    "small_pages": (config(32, 61, [
        layer(attention(6, 6, 16, 0.6, rot(2, 30.0), softcap=4.0), 24),
        layer(rglru(16, 2, 3), None),
        layer(latent(4, 8, 2, 24, 14, 0.7), 16),
        layer(attention(5, 1, 24, 0.5, rot(24, 1000.0, (1.0, 20, 2.0, 1.0))), 8),
    ]), 64, 4),
}


def _normal(generator, shape, std):
    return torch.randn(shape, generator=generator, dtype=torch.float32) * std


def make_weights(cfg: Mapping[str, Any], seed: int) -> dict[str, torch.Tensor]:
    """fp32 tensors whose values are exact in bfloat16 (a model folder written in either dtype holds the same numbers)."""
    g = torch.Generator().manual_seed(seed)
    width, vocab = cfg["width"], cfg["vocab"]

    def norm(size):
        return 1.0 + _normal(g, (size,), 0.2)

    w: dict[str, torch.Tensor] = {"embed": _normal(g, (vocab, width), 0.7), "embed.norm": norm(width), "final.norm": norm(width),
                                  "head": _normal(g, (vocab, width), width ** -0.5)}
    for index, entry in enumerate(cfg["layers"]):
        p, m, kind = f"l{index}", entry["mixer"], entry["type"]
        q = f"{p}.mix"
        w[f"{p}.norm1"] = norm(width)
        w[f"{p}.ls1"] = _normal(g, (width,), 0.3) + 0.8
        if kind == "attention":
            heads, kvh, dim = m["heads"], m["kv_heads"], m["dim"]
            w[f"{q}.q"] = _normal(g, (heads * dim, width), 1.3 * width ** -0.5)
            w[f"{q}.k"] = _normal(g, (kvh * dim, width), 1.1 * width ** -0.5)
            w[f"{q}.o"] = _normal(g, (width, heads * dim), (heads * dim) ** -0.5)
        elif kind == "latent_attention":
            heads, dim, r, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            gain = (2.5 / m["scale"]) ** 0.5 * (dim + r) ** -0.25  # scores of a few units
            w[f"{q}.q"] = _normal(g, (heads * (dim + r), width), gain * width ** -0.5)
            w[f"{q}.dkv"] = _normal(g, (rank + r, width), width ** -0.5)
            w[f"{q}.dkv"][rank:] *= gain
            w[f"{q}.dkv.norm"] = norm(rank)
            w[f"{q}.uk"] = _normal(g, (heads * dim, rank), gain * rank ** -0.5)
            w[f"{q}.uv"] = _normal(g, (heads * vdim, rank), rank ** -0.5)
            w[f"{q}.g"] = _normal(g, (heads * vdim, width), 1.5 * width ** -0.5)
            w[f"{q}.o"] = _normal(g, (width, heads * vdim), 1.5 * (heads * vdim) ** -0.5)
        else:
            inner, blocks, taps = m["width"], m["blocks"], m["conv"]
            n = inner // blocks
            for name in ("y", "x"):
                w[f"{q}.{name}"] = _normal(g, (inner, width), 1.2 * width ** -0.5)
                w[f"{q}.{name}.b"] = _normal(g, (inner,), 0.4)
            w[f"{q}.conv"] = _normal(g, (inner, taps), 0.6)
            w[f"{q}.conv.b"] = _normal(g, (inner,), 0.3)
            for name in ("ra", "ri"):
                w[f"{q}.{name}"] = _normal(g, (blocks, n, n), 1.5 * n ** -0.5)
                w[f"{q}.{name}.b"] = _normal(g, (blocks, n), 0.6)
            w[f"{q}.lam"] = _normal(g, (inner,), 2.0) - 2.5
            w[f"{q}.o"] = _normal(g, (width, inner), 2.0 * inner ** -0.5)
        if entry["mlp"] is None:
            continue
        ff = entry["mlp"]["ff"]
        w[f"{p}.norm2"] = norm(width)
        w[f"{p}.ls2"] = _normal(g, (width,), 0.3) + 0.8
        w[f"{p}.mlp.gate"] = _normal(g, (ff, width), 1.5 * width ** -0.5)
        w[f"{p}.mlp.up"] = _normal(g, (ff, width), 1.5 * width ** -0.5)
        w[f"{p}.mlp.down"] = _normal(g, (width, ff), ff ** -0.5)
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
