"""Replays a trace of token ids through a model, step by step, and writes logits (``bin/trace_run``).

Steps arrive on standard input, one JSON object per line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

The entries of a step run as one batch from the state that earlier steps left; ``want`` lists the places among an entry's
tokens whose logits are written, ``end`` the requests that give their memory back afterwards. A step with wanted places
writes ``<out>/<step>.f32`` (little-endian fp32, [wanted, vocab]); every step prints ``done <step>``. Nothing is sampled: the
steps go through the same runner, cache and kernels as the serving engine's (``serving.hybrid_runner.HybridRunner``)."""
from __future__ import annotations

import argparse
import json
import os
import sys

from ..ops.ragged import as_mask


def _cache_size(model, max_tokens: int):
    """State slots and cache blocks for ``max_tokens`` live tokens: a request holds at least one token, at most two partly
    filled blocks of tokens, and for masks that average older blocks at most one partly filled block of averages."""
    slots = max(1, min(max_tokens, 256))
    per_slot = 0
    for layer in model.layers:
        for shape, dt in layer.mixer.state_spec(model.act_dtype).values():
            n = dt.itemsize
            for s in shape:
                n *= s
            per_slot += n
    slots = max(1, min(slots, (8 << 30) // max(per_slot, 1)))
    pools = {as_mask(s[3]).pool for layer in model.layers for s in layer.mixer.kv_specs()} - {0}
    return slots, max_tokens // 16 + 2 * slots + sum(max_tokens // (16 * p) + slots for p in pools)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a token trace and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)

    import torch
    from .. import _build
    if not torch.cuda.is_available():
        print("trace_run: no CUDA device", file=sys.stderr)
        return 2
    _build.load_cuda(subset="hybrid")      # compiles only what hybrid decoders need when the full library is not built
    from ..hub.model_hub import ModelHub
    from ..ops._lib import check_status
    from .hybrid_runner import HybridRunner
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.set_float32_matmul_precision("highest")
    model = ModelHub.from_pretrained(a.model, dtype=getattr(torch, a.dtype), device="cuda")
    if not hasattr(model, "init_cache"):
        print(f"trace_run: {type(model).__name__} is not served by the hybrid runner", file=sys.stderr)
        return 2
    slots, blocks = _cache_size(model, max(1, a.max_tokens))
    runner = HybridRunner(model, model.init_cache(slots, blocks))
    runner.enable_graphs(min(slots, 32))
    seqs, next_id = {}, 0
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step.get("entries", ()):
            if e["id"] not in seqs:
                seqs[e["id"]] = next_id
                runner.cache.add_sequence(next_id)
                next_id += 1
            if e["tokens"]:
                entries.append((seqs[e["id"]], e["tokens"], e.get("want", ())))
        if entries:
            logits = runner.step(entries)
            if logits.shape[0]:
                out = logits.float().cpu().contiguous()
                check_status()
                with open(os.path.join(a.out, f"{step['step']}.f32"), "wb") as f:
                    f.write(out.numpy().astype("<f4", copy=False).tobytes())
        for rid in step.get("end", ()):
            if rid in seqs:
                runner.cache.free_sequence(seqs.pop(rid))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
