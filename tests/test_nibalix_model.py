"""Nibalix through the engine -- scheduler, paged rows, state slots, graphs -- against the plain oracle on whole sequences."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import nibalix_oracle as O
from jittorinfer_b200 import ops
from jittorinfer_b200.models import nibalix, registry
from jittorinfer_b200.runtime.engine import EngineConfig, LLMEngine
from jittorinfer_b200.runtime.sampling import SamplingParams
from nibalix_cases import CASES, config, gru, latent, moe, tokens, weights, write_model

GPU = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
WHERE = [pytest.param("cpu", F32, id="cpu"), pytest.param("cuda", F32, id="cuda-f32", marks=GPU),
         pytest.param("cuda", BF16, id="cuda-bf16", marks=GPU)]
EXACT = WHERE[:2]
_oracle = {}


def oracle(case, toks, cfg=None, w=None):
    key = (case, tuple(toks))
    if key not in _oracle:
        cfg = cfg or CASES[case]
        with torch.no_grad():
            _oracle[key] = O.forward(cfg, w or weights(cfg), toks)
    return _oracle[key]


def engine(case, dev, dtype, n_ctx=1024, n_parallel=4, cfg=None, w=None, **kw):
    cfg = cfg or CASES[case]
    hp = nibalix.NibalixHParams.from_config(cfg)
    m = nibalix.NibalixModel(hp, (w or weights(cfg)).items(), dtype=dtype, device=dev, max_positions=n_ctx)
    kw.setdefault("n_batch", n_ctx)
    kw.setdefault("graph_buckets", (1, 2, 4))
    return LLMEngine(m, EngineConfig(n_ctx=n_ctx, n_parallel=n_parallel, n_ctx_slot=kw.pop("n_ctx_slot", n_ctx), **kw))


def check(got, want, dtype, what=""):
    """Per row: centred error over the vocabulary against the size of the logits.  bf16: a row whose expert choice sits on a
    near-tie may move; nearly all rows must be tight."""
    d = (got - want).double()
    d = d - d.mean(-1, keepdim=True)
    err = d.pow(2).mean(-1).sqrt() / want.double().std()
    if dtype == F32:
        assert err.max() < 1e-4, f"{what}: row {int(err.argmax())} is off by {err.max():.2e}"
    else:
        assert err.median() < 0.02 and (err < 0.05).double().mean() >= 0.9, f"{what}: median {err.median():.3f}, worst {err.max():.3f}"


def feed_all(eng, key, toks, cuts):
    """Feeds a sequence in portions, all logits wanted."""
    out, p, k = [], 0, 0
    while p < len(toks):
        n = min(cuts[k % len(cuts)], len(toks) - p)
        out.append(eng.feed([(key, toks[p:p + n], range(n))]))
        p, k = p + n, k + 1
    return torch.cat(out)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("case", list(CASES))
def test_prompt_portions_and_single_tokens_give_the_same_logits(case, dev, dtype):
    toks = tokens(CASES[case], 150)
    want = oracle(case, toks)
    eng = engine(case, dev, dtype)
    for cuts in ([150], [64], [2], [37, 2, 3], [1], [129, 1, 1, 5]):
        check(feed_all(eng, "s", toks, cuts), want, dtype, f"{case} {cuts}")
        eng.end_feed("s")
    assert eng.kv.used_blocks == 0 and eng.kv.check()
    if dev == "cuda":
        assert eng.stats["graph_steps"] >= 150
        ops.nat().check_status()


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_unequal_requests_in_one_batch_with_blocks_and_slots_used_again(dev, dtype):
    """Eight sequences through four slots and a pool that never holds more than what lives: portions of some beside single
    tokens of others, sequences left out of steps, slots and blocks passed on at once."""
    case = "mixed"
    lens = [150, 70, 3, 129, 64, 1, 200, 90]
    seqs = {i: tokens(CASES[case], n, seed=20 + i) for i, n in enumerate(lens)}
    eng = engine(case, dev, dtype, n_ctx=640)
    g = torch.Generator().manual_seed(0)
    got = {i: [] for i in seqs}
    at, live, waiting = {i: 0 for i in seqs}, [], list(seqs)
    need = lambda: sum((lens[i] + 63) // 64 for i in live)           # noqa: E731
    while live or waiting:
        while waiting and len(live) < 4 and need() + (lens[waiting[0]] + 63) // 64 <= 10:
            live.append(waiting.pop(0))
        entries = []
        for i in live:
            r = int(torch.randint(0, 5, (1,), generator=g))
            n = min([0, 1, 1, 2, 40][r], lens[i] - at[i])
            if n:
                entries.append((i, seqs[i][at[i]:at[i] + n], range(n)))
                at[i] += n
        out = eng.feed(entries)
        k = 0
        for i, t, _ in entries:
            got[i].append(out[k:k + len(t)])
            k += len(t)
        for i in [i for i in live if at[i] == lens[i]]:
            eng.end_feed(i)
            live.remove(i)
    for i in seqs:
        check(torch.cat(got[i]), oracle(case, seqs[i]), dtype, f"sequence {i}")
    assert eng.kv.used_blocks == 0


@pytest.mark.parametrize("dev,dtype", EXACT)
def test_long_decoding_keeps_the_state(dev, dtype):
    """300 single tokens with a recurrence that forgets slowly, windows passed several times."""
    cfg = config([gru(32), latent(window=50), dict(latent(window=90, kv_from=1), mlp=None)], width=32, vocab=90, mlp=moe(16, 3, 1))
    w = weights(cfg, seed=3)
    w["l0.mix.z.b"] -= 4
    toks = tokens(cfg, 330)
    want = oracle("slow", toks, cfg, w)
    eng = engine(None, dev, dtype, cfg=cfg, w=w)
    check(feed_all(eng, 0, toks, [30] + [1] * 300), want, dtype)


@pytest.mark.parametrize("dev,dtype", EXACT)
@pytest.mark.parametrize("window", [63, 64, 65])
@pytest.mark.parametrize("decode", [False, True])
def test_the_windows_edge_shows(dev, dtype, window, decode):
    """One token's key stands out in an attention-only model: positions that still see it and the first that does not, in a
    prompt and in decoding, at block borders.  (The oracle itself is shown to be sensitive to a window that is one off.)"""
    cfg = config([latent(window=window, heads=2, dim=16, rot=2, base=1e9, rank=24)], width=32, vocab=60, mlp=None, taps=1, mult=1.0)
    w = weights(cfg, seed=5)
    w["embed"][7] = w["embed"][7] * 0 + w["embed"][9]                # token 7: a copy of 9 whose key is ...
    hot = torch.zeros(32)
    hot[3] = 6.0
    w["embed"][7] += hot                                             # ... along one direction every query likes
    w["l0.mix.dkv"][:24] *= 0.3
    w["l0.mix.dkv"][0] = 0
    w["l0.mix.dkv"][0, 3] = 4.0
    w["l0.mix.uk"][:, 0] = 1.5
    w["l0.mix.q"][:, :] *= 0.2
    w["l0.mix.q"][:, 5] = 1.0
    w["embed"][:, 5] = 3.0
    toks = [t if t != 7 else 8 for t in tokens(cfg, 3 * window, seed=2)]
    toks[20] = 7
    want = oracle(("edge", window), toks, cfg, w)
    off = json.loads(json.dumps(cfg))
    off["layers"][0]["mixer"]["mask"]["size"] = window + 1
    moved = (oracle(("edge+1", window), toks, off, w) - want).abs().amax(-1)
    assert moved[20 + window] > 0.03 and moved[19 + window] < 0.1 * moved[20 + window]    # the first position that must not see token 20
    eng = engine(None, dev, dtype, cfg=cfg, w=w)
    check(feed_all(eng, 0, toks, [1] if decode else [len(toks)]), want, dtype)


# ---- the generation path ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", EXACT)
@pytest.mark.parametrize("run_ahead", [False, True])
def test_greedy_generation_through_the_scheduler(dev, dtype, run_ahead):
    """More requests than slots, prompts in portions beside decoding sequences, a pool small enough to preempt."""
    case = "mixed"
    cfg, w = CASES[case], weights(CASES[case])
    prompts = [tokens(cfg, n, seed=40 + n) for n in (70, 5, 1, 100, 33, 64)]
    eng = engine(case, dev, dtype, n_ctx=320, n_parallel=3, n_batch=48, n_ctx_slot=192, run_ahead=run_ahead)
    outs = eng.generate(prompts, SamplingParams(temperature=0.0, ignore_eos=True), max_new_tokens=24)
    for p, out in zip(prompts, outs):
        lg = O.forward(cfg, w, p + out)[len(p) - 1:-1]               # one pass: every generated id is the best (or a tie within rounding)
        best = lg.max(-1).values
        assert len(out) == 24 and bool((best - lg[torch.arange(24), torch.tensor(out)] < 1e-3).all()), (len(p), out)
    assert eng.kv.check()


@pytest.mark.parametrize("dev,dtype", EXACT)
def test_a_conversation_continues_and_a_cut_prefix_starts_over(dev, dtype):
    """A prompt that extends everything a slot holds continues from its state; one that shares only a part of it (or is shorter)
    is evaluated from the start, because the state exists at the end only; blocks are never shared between slots."""
    case = "mixed"
    cfg, w = CASES[case], weights(CASES[case])
    eng = engine(case, dev, dtype, n_parallel=2)
    sp = SamplingParams(temperature=0.0, ignore_eos=True, max_tokens=6)

    def run(prompt):
        before = eng.stats["tokens_in"]
        out = eng.generate([prompt], sp)[0]
        lg = O.forward(cfg, w, prompt + out)[len(prompt) - 1:-1]
        assert bool((lg.max(-1).values - lg[torch.arange(6), torch.tensor(out)] < 1e-3).all())
        return out, eng.stats["tokens_in"] - before

    first = tokens(cfg, 90, seed=7)
    out, n = run(first)
    assert n == 95                                                   # 90 + 5 fed back
    longer = first + out[:5] + tokens(cfg, 12, seed=8)
    _, n = run(longer)
    assert n == 12 + 5                                               # continued from the state
    _, n = run(first)                                                # a proper prefix of what the slot holds
    assert n == 95
    _, n = run(first[:70] + tokens(cfg, 9, seed=9))                  # shares 70 tokens with both slots
    assert n == 79 + 5
    assert eng.sched.stats()["prefix_shared"] == 0


def test_sampling_modes_cancel_reset_and_state_isolation():
    case = "mixed"
    eng = engine(case, "cpu", F32, n_parallel=2)
    sp = SamplingParams(temperature=0.9, top_k=20, seed=3, max_tokens=8, ignore_eos=True)
    a = eng.generate([[1, 2, 3]], sp)
    rid = eng.add_request(tokens(CASES[case], 40), SamplingParams(temperature=0.0, ignore_eos=True, max_tokens=50))
    for _ in range(5):
        eng.step()
    assert eng.cancel(rid)
    assert eng.generate([[1, 2, 3]], sp) == a
    eng.reset()
    assert eng.generate([[1, 2, 3]], sp) == a


def test_feed_and_generate_share_an_engine():
    case = "mixed"
    toks = tokens(CASES[case], 100)
    eng = engine(case, "cpu", F32, n_ctx=256, n_parallel=2)
    got = [eng.feed([("x", toks[:50], range(50))])]
    out = eng.generate([toks[:20]], SamplingParams(temperature=0.0, ignore_eos=True), max_new_tokens=3)[0]
    assert len(out) == 3
    got.append(eng.feed([("x", toks[50:], range(50))]))
    check(torch.cat(got), oracle(case, toks), F32)
    with pytest.raises(RuntimeError):                                # 256 cached tokens, 100 held by x
        eng.feed([("y", tokens(CASES[case], 200), [])])
    with pytest.raises(ValueError):
        eng.feed([("x", [1], [1])])
    with pytest.raises(ValueError):
        eng.feed([("x", [10 ** 6], [])])
    eng.end_feed("x")
    eng.end_feed("y")
    assert not eng.has_work()


# ---- files, registry, command lines -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
def test_folder_model_through_the_registry_and_the_trace_runner(tmp_path, dev, dtype):
    case = "mixed"
    cfg, w = CASES[case], weights(CASES[case])
    d = write_model(tmp_path / "m", cfg, w)
    assert registry.for_path(d).name == "Nibalix" and nibalix.load_config(d).to_config()["layers"] == cfg["layers"]
    toks = {"a": tokens(cfg, 80, seed=1), "b": tokens(cfg, 40, seed=2)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks["a"][:70], "want": [0, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": toks["b"], "want": []}, {"id": "a", "tokens": toks["a"][70:71], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": toks["a"][71:72], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "b", "tokens": toks["b"][:3], "want": [2]}, {"id": "a", "tokens": toks["a"][72:], "want": [7]}],
              "end": ["a", "b"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "bfloat16" if dtype == BF16 else "float32",
                        "--out", str(out), "--max-tokens", "192", "--device", dev], input="\n".join(map(json.dumps, steps)) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.split("\n") if x.startswith("done ")] == ["done 0", "done 1", "done 2", "done 3"]
    read = lambda n: torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())      # noqa: E731
    la, lb = oracle(case, toks["a"]), oracle(case, toks["b"])
    got = torch.cat([read(0), read(1), read(3)])
    check(got, torch.stack([la[0], la[69], la[70], lb[2], la[79]]), dtype)
    assert not (out / "2.f32").exists()


def test_configuration_and_checkpoint_errors(tmp_path):
    cfg, w = CASES["mixed"], weights(CASES["mixed"])
    load = nibalix.NibalixHParams.from_config
    for edit in (lambda c: c["layers"][3]["mixer"].update(kv_from=3), lambda c: c["layers"][3]["mixer"].update(kv_from=0),
                 lambda c: c["layers"][3]["mixer"].update(kv_rank=9), lambda c: c["layers"][0].update(type="other"),
                 lambda c: c["layers"][0]["mlp"].update(kind="dense"), lambda c: c.update(architecture="Other"),
                 lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4), lambda c: c["layers"][1]["mixer"]["mask"].update(size=0)):
        c = json.loads(json.dumps(cfg))
        edit(c)
        with pytest.raises(ValueError):
            load(c)
    hp = load(cfg)
    short = dict(list(w.items())[:-1])
    with pytest.raises(KeyError):
        list(nibalix.iter_checkpoint(write_model(tmp_path / "a", cfg, short), hp))
    with pytest.raises(ValueError):
        list(nibalix.iter_checkpoint(write_model(tmp_path / "b", cfg, dict(w, extra=w["head"])), hp))
    with pytest.raises(ValueError):
        list(nibalix.iter_checkpoint(write_model(tmp_path / "c", cfg, dict(w, head=w["head"][:-1])), hp))
    with pytest.raises(ValueError):
        registry.for_path(write_model(tmp_path / "d", dict(cfg, architecture="Other"), w))
    from jittorinfer_b200.runtime.factory import build_engine
    with pytest.raises(ValueError):
        build_engine(hp, device="cpu", world=2)


def test_generate_command_line_serves_a_folder(tmp_path, capsys):
    from jittorinfer_b200 import generate
    cfg, w = CASES["mixed"], weights(CASES["mixed"])
    d = write_model(tmp_path / "m", cfg, w)
    prompt = tokens(cfg, 9, seed=3)
    assert generate.main(["--model", d, "--tokens", ",".join(map(str, prompt)), "-n", "5", "--json", "--device", "cpu"]) == 0
    out = json.loads(capsys.readouterr().out.strip().split("\n")[-1])
    assert out["completions"][0]["tokens"] == O.generate(cfg, w, prompt, 5)
    assert registry.preset("nibalix-tiny").n_layer == 4 and registry.preset("tiny").n_layer == 2


@pytest.mark.parametrize("dev,dtype", EXACT)
def test_defragmentation_moves_rows_of_every_width(dev, dtype):
    case = "mixed"
    toks = {k: tokens(CASES[case], 150, seed=k) for k in (1, 2)}
    eng = engine(case, dev, dtype, n_ctx=640)
    eng.feed([(0, tokens(CASES[case], 130), [])])
    got = {k: [eng.feed([(k, toks[k][:100], range(100))])] for k in toks}
    eng.end_feed(0)                                                  # holes below the two that live
    assert eng.defrag(16) > 0 and eng.kv.check()
    for k in toks:
        got[k].append(eng.feed([(k, toks[k][100:], range(50))]))
        check(torch.cat(got[k]), oracle(case, toks[k]), dtype, f"sequence {k}")


@GPU
@pytest.mark.parametrize("window", [64, 130, 300])
def test_tensor_core_attention_shapes_in_the_model(window):
    """Head sizes of the tcgen05 attention kernels: prompts in the per-head form, short portions and decoding in the absorbed
    form, a layer on another layer's rows."""
    big = dict(heads=2, dim=128, rot=64, vdim=128, rank=512, base=10000.0)
    cfg = config([gru(128), latent(window=window, **big), latent(window=2 * window, kv_from=1, **dict(big, heads=3))], width=256, vocab=500,
                 mlp=moe(64, 8, 2))
    w = weights(cfg, seed=1)
    toks = tokens(cfg, 330)
    want = oracle(("wide", window), toks, cfg, w)
    eng = engine(None, "cuda", BF16, cfg=cfg, w=w)
    n0 = dict(ops.nat().launches_by_name)
    for cuts in ([330], [200, 70, 60], [100, 9, 2, 30], [290] + [1] * 40):
        check(feed_all(eng, 0, toks, cuts), want, BF16, f"{cuts}")
        eng.end_feed(0)
    ops.nat().check_status()
    ran = {k: ops.nat().launches_by_name.get(k, 0) - n0.get(k, 0) for k in ("mha_prefill", "mla_flash", "mla_attention", "mingru", "block_update")}
    assert ran["mha_prefill"] > 0 and ran["mla_flash"] > 0 and ran["mla_attention"] == 0 and ran["mingru"] > 0, ran
