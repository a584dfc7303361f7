"""``bench.py --design koravik``: prefill and decode throughput of the Koravik design at a few layer sizes, beside the closest
model this package has at equal size: Mapalorn with grouped-query attention in every layer (looped layers, score-routed
experts beside a shared expert) of the same width, layer runs, heads, key/value heads and bytes of expert weights (random
bf16 weights, synthetic tokens).  One JSON line; the default workload of bench.py and its line are untouched by this option.

Six layers of which the first two run twice: eight layer runs.  Heads of 128, all columns rotated; Koravik's window keeps
1,024 positions and the first 4.  Koravik's experts have two matrices where Mapalorn's have three, so they have half as
many rows again.  Measured as ``bench_makilorn.py`` measures: a 2,048-token prompt in one step (median of 5 after 3 warm-up
steps) and decode steps at batch 8 and 64 over 2,048-token prompts (CUDA events around ``steps`` replayed steps after
``warmup``; every step reads its layers' weights and the requests' caches, several times the 126 MB L2).
"""

from __future__ import annotations

import json
import sys

from bench_makilorn import LAYERS, PAGE_SIZE, PROMPT, VOCAB, _decode_ms, _engine, _prefill_ms

# width, heads, key/value heads, experts, experts a token, rows of a gated expert and of the gated shared expert
SIZES = {
    "w2048": dict(width=2048, heads=16, kv_heads=4, experts=32, top=4, ff=1024, shared=1024),
    "w4096": dict(width=4096, heads=32, kv_heads=4, experts=32, top=4, ff=2048, shared=2048),
}
LOOP = {"start": 0, "stop": 2, "times": 2}
LISTED = 6
WINDOW, KEPT = 1024, 4


def koravik_config(size: dict) -> dict:
    mixer = {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
             "rot": {"base": 500000.0, "dims": 128}, "mask": {"size": WINDOW, "keep_first": KEPT}}
    mlp = {"kind": "moe", "router": {"experts": size["experts"], "top": size["top"]}, "expert": {"ff": size["ff"] * 3 // 2}, "shared": {"ff": size["shared"] * 3 // 2}}
    return {"architecture": "Koravik", "vocab": VOCAB, "width": size["width"], "norm": {"eps": 1e-6}, "residual_mult": 0.4, "logit_scale": 0.25,
            "max_positions": 4096, "loop": LOOP, "layers": [{"type": "attention", "mixer": mixer, "mlp": mlp}] * LISTED}


def mapalorn_config(size: dict) -> dict:
    mixer = {"heads": size["heads"], "kv_heads": size["kv_heads"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": {"base": 500000.0, "dims": 128}}
    mlp = {"kind": "moe", "router": {"experts": size["experts"], "top": size["top"]}, "expert": {"ff": size["ff"]}, "shared": {"ff": size["shared"]}}
    return {"architecture": "Mapalorn", "vocab": VOCAB, "width": size["width"], "norm": {"eps": 1e-6}, "max_positions": 4096, "loop": LOOP,
            "layers": [{"type": "attention", "mixer": mixer, "mlp": mlp}] * LISTED}


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
        for model, config in (("koravik", koravik_config(size)), ("mapalorn", mapalorn_config(size))):
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
        for what in ("prefill", "decode_b8", "decode_b64"):
            entry[f"{what}_ratio"] = entry["koravik"][f"{what}_tokens_per_s"] / entry["mapalorn"][f"{what}_tokens_per_s"]
        sizes[name] = dict(size, layer_runs=LAYERS, window=WINDOW, keep_first=KEPT, **entry)
    print(json.dumps({
        "metric": "koravik_vs_mapalorn_tokens_per_s", "design": "Koravik", "n_gpus": 1, "steps": steps, "warmup": warmup, "dtype": "bf16",
        "data": "synthetic", "gpu_launches": launches,
        "config": {"prompt_len": PROMPT, "page_size": PAGE_SIZE, "layer_runs": LAYERS, "inputs": "weights and caches larger than L2"},
        "sizes": sizes,
    }))
    return 0
