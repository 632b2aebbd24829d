"""Trace replay: ``bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps``.

Feeds given token ids through the serving engine step by step (``LLMEngine.feed``: its scheduler, cache, state slots, CUDA
graphs and kernels) and writes the logits asked for; nothing is sampled.  Standard input carries one step per line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step form one batch.  The logits at the wanted places, in the order of the entries and of ``want``, go to
``<out>/<step>.f32`` as little-endian fp32 [wanted, vocab]; ``done <step>`` is printed after every step.  ``end`` names the
requests whose slot and cache blocks are given back after the step.  ``--max-tokens`` sizes the cache pool: the most tokens live
requests hold at any time, each rounded up to whole cache blocks.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

BLOCK = 64


def build(model: str, dtype: str, max_tokens: int, n_seqs: int = 4, device=None):
    """The serving engine of a model folder (or GGUF file) with a pool of ``max_tokens`` cached tokens."""
    import torch

    from .runtime.factory import build_engine
    dev = torch.device(device or "cuda")
    if dtype == "float32":                      # true 32-bit products
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cudnn.allow_tf32 = False
    n = max(BLOCK, (max_tokens + BLOCK - 1) // BLOCK * BLOCK)
    buckets = tuple(b for b in (1, 2, 4, 8, 16, 32, 64) if b < n_seqs) + (n_seqs,)
    return build_engine(None, gguf_path=model, device=dev, dtype=getattr(torch, dtype), n_parallel=n_seqs, n_ctx=n, n_ctx_slot=n, n_batch=n,
                        graph_buckets=buckets)


def replay(eng, lines, out_dir: str, emit=print) -> None:
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]]
        logits = eng.feed(entries)
        if logits.shape[0]:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4", copy=False).tobytes())
            os.replace(path + ".part", path)
        for key in step.get("end", []):
            eng.end_feed(key)
        emit(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="cached tokens the pool holds")
    ap.add_argument("--device", default=None, help="cuda (default) | cpu: the reference ops, for debugging without a GPU")
    a = ap.parse_args(argv)
    os.makedirs(a.out, exist_ok=True)
    eng = build(a.model, a.dtype, a.max_tokens, device=a.device)
    replay(eng, sys.stdin, a.out, lambda s: print(s, flush=True))
    return 0


if __name__ == "__main__":
    sys.exit(main())
