"""Prefill and decode throughput of one design beside the engine's closest other model at equal layer sizes.

Called by ``bench.py --design NAME``.  Random weights, random token ids, one GPU.  For every size both models run the same work
through the engine's public step functions: prompts of ``--prompt-len`` tokens in one portion each (``LLMEngine.feed`` with the
last token's logits wanted), then decode steps (``LLMEngine.step``) at several numbers of concurrent sequences, CUDA-graph
replays included.  Times are CUDA-event times of whole steps on the launching stream, host work between launches included.  The
weights exceed the L2 many times over, so no flush is needed.
"""
from __future__ import annotations

import json
import statistics
import time

import torch


def sizes(design: str):
    """(label, hyper-parameters of the design, of the closest model) with equal widths, heads, experts, layers and vocabulary."""
    from ..models.hparams import DeepSeek2HParams
    from ..models.registry import preset
    if design == "lugovik":
        dense = lambda n, d, h, ff: DeepSeek2HParams(n_layer=n, n_layer_dense_lead=n, n_embd=d, n_head=h, n_ff=ff)       # noqa: E731
        return [("width 2048, 16 heads of 128, feed-forward 5632, 12 layers", preset("lugovik-lite"), dense(12, 2048, 16, 5632)),
                ("width 4096, 32 heads of 128, feed-forward 11008, 8 layers", preset("lugovik-wide"), dense(8, 4096, 32, 11008))]
    if design in ("zomavik", "rupatar"):
        runs = "layer runs" if design == "zomavik" else "layers"
        v2 = DeepSeek2HParams(n_layer=4, n_layer_dense_lead=0, n_embd=5120, n_head=128, n_ff_exp=1536, n_expert=160, expert_weights_scale=16.0,
                              n_group=8, topk_group=3, q_lora_rank=1536)
        return [(f"width 2048, 16 heads, 64 experts top-6 of 1408 + 2 shared, 12 {runs}", preset(f"{design}-lite"),
                 DeepSeek2HParams(n_layer=12, n_layer_dense_lead=0)),
                (f"width 5120, 40 heads (closest: 128), 160 experts top-6 of 1536 + 2 shared, 4 {runs}", preset(f"{design}-v2"), v2)]
    if design != "nibalix":
        raise SystemExit(f"unknown design {design!r} (known: nibalix, lugovik, zomavik, rupatar)")
    lite = DeepSeek2HParams(n_layer=12, n_layer_dense_lead=0, n_expert_shared=0)
    v2 = DeepSeek2HParams(n_layer=4, n_layer_dense_lead=0, n_expert_shared=0, n_embd=5120, n_head=128, n_ff_exp=1536, n_expert=160,
                          expert_weights_scale=16.0, n_group=8, topk_group=3, q_lora_rank=1536)
    return [("width 2048, 16 heads, 64 experts top-6 of 1408, 12 layers", preset("nibalix-lite"), lite),
            ("width 5120, 128 heads, 160 experts top-6 of 1536, 4 layers", preset("nibalix-v2"), v2)]


def measure(hp, prompt_len: int, concurrency, steps: int, warmup: int, note=lambda s: None) -> dict:
    from .. import ops
    from ..runtime.factory import build_engine
    from ..runtime.sampling import SamplingParams
    ctx = prompt_len + 2 * steps + warmup + 64
    n = max(concurrency)
    eng = build_engine(hp, device="cuda", n_parallel=n, n_ctx_slot=(ctx + 63) // 64 * 64, n_batch=max(2048, prompt_len), graph_buckets=tuple(concurrency))
    g = torch.Generator().manual_seed(1)
    rnd = lambda k: torch.randint(0, hp.n_vocab, (k,), generator=g).tolist()        # noqa: E731
    out = {"weight_gib": round(eng.model.weight_bytes() / 2 ** 30, 2), "layers": hp.n_layer}

    def timed(fn):
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1)

    ms = []
    for i in range(warmup + steps // 4):
        toks = rnd(prompt_len)
        t = timed(lambda: eng.feed([("p", toks, [prompt_len - 1])]))                 # noqa: B023
        eng.end_feed("p")
        if i >= warmup:
            ms.append(t)
    med = statistics.median(ms)
    out["prefill"] = {"tokens": prompt_len, "ms": round(med, 3), "tokens_per_s": round(prompt_len / med * 1e3, 1)}
    note(f"prefill {med:.2f} ms")
    out["decode"] = {}
    for c in concurrency:
        sp = SamplingParams(max_tokens=2 * steps + warmup + 8, ignore_eos=True)
        ids = [eng.add_request(rnd(prompt_len), sp) for _ in range(c)]
        while any(not eng.requests[i].output for i in ids):
            eng.step()
        for _ in range(warmup):
            eng.step()
        l0 = eng.launches
        regions = [timed(lambda: [eng.step() for _ in range(steps)]) / steps for _ in range(1)]
        launches = (eng.launches - l0) // steps
        graph = eng._graphs.get((c, "greedy"))
        gms = None
        if graph is not None:                     # the step's device time alone (the sequences are not read afterwards)
            gms = timed(lambda: [graph[0].replay() for _ in range(16)]) / 16         # noqa: B023
        for i in ids:
            eng.cancel(i)
            eng.requests.pop(i, None)
        eng.reset()
        med = statistics.median(regions)
        out["decode"][str(c)] = {"ms_per_step": round(med, 4), "tokens_per_s": round(c / med * 1e3, 1), "launches_per_step": launches,
                                 "graph_ms": None if gms is None else round(gms, 4)}
        note(f"decode x{c}: {med:.3f} ms")
    ops.nat().check_status()
    del eng
    torch.cuda.empty_cache()
    return out


def run(args, sampler=None) -> int:
    t0 = time.time()

    def note(msg):
        import sys
        print(f"[design +{time.time() - t0:6.1f}s] {msg}", file=sys.stderr, flush=True)
    recs, launches = [], 0
    for label, hp, near in sizes(args.design):
        rec = {"size": label}
        for name, h in ((args.design, hp), ("closest", near)):
            note(f"{label}: {name}")
            rec[name] = measure(h, args.prompt_len, (1, 8, 64), args.steps, max(3, args.warmup), note)
            launches += sum(v["launches_per_step"] * args.steps for v in rec[name]["decode"].values())
        a, b = rec[args.design], rec["closest"]
        rec["time_ratio"] = {"prefill": round(a["prefill"]["ms"] / b["prefill"]["ms"], 3),
                             **{f"decode_{c}": round(a["decode"][c]["ms_per_step"] / b["decode"][c]["ms_per_step"], 3) for c in a["decode"]}}
        recs.append(rec)
    head = recs[0][args.design]["decode"]["8"]
    out = {"metric": f"{args.design}: decode output tokens/s at concurrency 8, first size", "value": head["tokens_per_s"], "unit": "tokens/s",
           "n_gpus": 1, "steps": args.steps, "warmup": max(3, args.warmup), "ms_per_step": head["ms_per_step"], "higher_is_better": True,
           "vs_baseline": None, "dtype": "bf16", "data": "synthetic (uniform-random token ids, random weights)", "impl": "ours",
           "config": {"prompt_len": args.prompt_len, "closest": "DeepSeek-V2 layers of equal sizes" + {"lugovik": ", dense feed-forwards", "nibalix": ", no shared experts"}.get(args.design, ""),
                      "l2": "weights exceed L2; no flush needed"},
           "gpu_launches": launches, "sizes": recs}
    if sampler is not None:
        out["clocks"] = sampler.stop()
    print(json.dumps(out))
    return 0
