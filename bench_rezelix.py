"""``bench.py --design rezelix``: prefill and decode throughput of the Rezelix design at a few layer sizes, beside the closest
model this package has at equal size, Tapasun (attention and recurrent layers with a short convolution, a silu-gated
feed-forward in each), and beside the dense Qwen3 decoder, all of the same width, layer count, heads, key/value heads and
feed-forward rows (random bf16 weights, synthetic tokens).  One JSON line; the default workload of bench.py and its line
are untouched by this option.

Eight layers: attention, latent attention, two recurrent ones, twice; Tapasun runs attention where this design runs either
attention and its state-space layer where this design recurs.  Attention heads of 128 with a quarter as many key/value
heads, all columns rotated (half of them in Tapasun); latent rows of 192 and 64 rotated columns; the recurrent unit as wide
as the model, in as many parts as there are heads, four taps.  Measured as ``bench_makilorn.py`` measures: a 2,048-token
prompt in one step (median of 5 after 3 warm-up steps) and decode steps at batch 8 and 64 over 2,048-token prompts (CUDA
events around ``steps`` replayed steps after ``warmup``; every step reads its layers' weights and the requests' caches,
several times the 126 MB L2).
"""

from __future__ import annotations

import json
import sys

from bench_makilorn import LAYERS, PAGE_SIZE, PROMPT, VOCAB, _decode_ms, _engine, _prefill_ms
from bench_tapasun import dense_config

SIZES = {
    "w2048": dict(width=2048, heads=16, ff=8192),
    "w4096": dict(width=4096, heads=32, ff=14336),
}
ORDER = ("attention", "latent_attention", "rglru", "rglru") * 2
assert len(ORDER) == LAYERS


def rezelix_config(size: dict) -> dict:
    width, heads = size["width"], size["heads"]
    scaling = {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}
    mixers = {
        "attention": {"heads": heads, "kv_heads": max(heads // 4, 1), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 50.0,
                      "rot": {"base": 500000.0, "dims": 128, "scaling": scaling}},
        "latent_attention": {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 192, "scale": 192 ** -0.5,
                             "rot": {"base": 500000.0, "dims": 64, "scaling": scaling}},
        "rglru": {"width": width, "blocks": heads, "conv": 4},
    }
    return {"architecture": "Rezelix", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6}, "max_positions": 4096,
            "layers": [{"type": kind, "mixer": mixers[kind], "mlp": {"kind": "dense", "ff": size["ff"]}} for kind in ORDER]}


def tapasun_config(size: dict) -> dict:
    width, heads = size["width"], size["heads"]
    rot = {"base": 500000.0, "dims": 64, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    attention = {"heads": heads, "kv_heads": max(heads // 4, 1), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": rot}
    space = {"heads": 2 * width // 64, "vdim": 64, "state": 128, "groups": 8, "norm_groups": 8, "conv": 4}
    layers = [("mamba2", space) if kind == "rglru" else ("attention", attention) for kind in ORDER]
    return {"architecture": "Tapasun", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5},
            "max_positions": 4096, "layers": [{"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": size["ff"]}} for kind, mixer in layers]}


def run(args) -> int:
    import torch

    if not torch.cuda.is_available():
        print("bench.py: no CUDA device; kairyu_b200 has no CPU path", file=sys.stderr)
        return 1
    torch.cuda.set_device(0)
    steps, warmup = min(args.steps, 64), max(args.warmup, 3)
    sizes = {}
    launches = 0
    for name, size in SIZES.items():
        entry = {}
        for model, config in (("rezelix", rezelix_config(size)), ("tapasun", tapasun_config(size)), ("dense", dense_config(size))):
            engine = _engine(config, 64)
            prefill = _prefill_ms(engine)
            result = {"prefill_ms": prefill, "prefill_tokens_per_s": PROMPT / (prefill / 1e3),
                      "weight_bytes_per_decode_token": engine.model.bytes_streamed_per_step()}
            for batch in (8, 64):
                ms, count = _decode_ms(engine, batch, steps, warmup)
                launches += count
                result[f"decode_b{batch}_ms"] = ms
                result[f"decode_b{batch}_tokens_per_s"] = batch / (ms / 1e3)
            entry[model] = result
            del engine
            torch.cuda.empty_cache()
        for other in ("tapasun", "dense"):
            for what in ("prefill", "decode_b8", "decode_b64"):
                entry[f"{what}_ratio_to_{other}"] = entry["rezelix"][f"{what}_tokens_per_s"] / entry[other][f"{what}_tokens_per_s"]
        sizes[name] = dict(size, layers=LAYERS, **entry)
    print(json.dumps({
        "metric": "rezelix_vs_tapasun_tokens_per_s", "design": "Rezelix", "n_gpus": 1, "steps": steps, "warmup": warmup, "dtype": "bf16",
        "data": "synthetic", "gpu_launches": launches,
        "config": {"prompt_len": PROMPT, "page_size": PAGE_SIZE, "layers": LAYERS, "inputs": "weights and caches larger than L2"},
        "sizes": sizes,
    }))
    return 0
