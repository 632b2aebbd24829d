"""Lugovik through the engine -- scheduler, paged rows, state slots, graphs -- against the plain oracle on whole sequences."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import lugovik_oracle as O
from jittorinfer_b200 import ops
from jittorinfer_b200.models import lugovik, registry
from jittorinfer_b200.runtime.engine import EngineConfig, LLMEngine
from jittorinfer_b200.runtime.sampling import SamplingParams
from lugovik_cases import CASES, config, delta, mamba, parallel, tokens, weights, write_model

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


def noise(case, toks, cfg=None, w=None):
    """How far the logits of each position move when every weight is off by about one bf16 rounding: what a bf16 run may differ by.
    (A read-out that is close to zero is all rounding once it is normed.)"""
    key = (case, tuple(toks), "noise")
    if key not in _oracle:
        cfg = cfg or CASES[case]
        g = torch.Generator().manual_seed(1)
        moved = {k: t * (1 + 2.0 ** -8 * torch.randn(t.shape, generator=g)) for k, t in (w or weights(cfg)).items()}
        with torch.no_grad():
            _oracle[key] = rows_off(O.forward(cfg, moved, toks), oracle(case, toks, cfg, w))
    return _oracle[key]


def rows_off(got, want):
    """Per row: centred difference over the vocabulary against the size of the logits."""
    d = (got - want).double()
    return (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().std()


def engine(case, dev, dtype, n_ctx=1024, n_parallel=4, cfg=None, w=None, **kw):
    cfg = cfg or CASES[case]
    hp = lugovik.LugovikHParams.from_config(cfg)
    m = lugovik.LugovikModel(hp, (w or weights(cfg)).items(), dtype=dtype, device=dev, max_positions=n_ctx)
    kw.setdefault("n_batch", n_ctx)
    kw.setdefault("graph_buckets", (1, 2, 4))
    return LLMEngine(m, EngineConfig(n_ctx=n_ctx, n_parallel=n_parallel, n_ctx_slot=kw.pop("n_ctx_slot", n_ctx), **kw))


def check(got, want, dtype, what="", off=None):
    """``off``: what rounding may do (``noise``), for bf16."""
    err = rows_off(got, want)
    if dtype == F32:
        assert err.max() < 1e-4, f"{what}: row {int(err.argmax())} is off by {err.max():.2e}"
    else:
        lim = 0.03 + 3 * off
        bad = int((err > lim).sum())
        assert bad <= max(1, len(err) // 20) and bool((err < 4 * lim).all()), f"{what}: median {err.median():.3f}, worst {(err / lim).max():.3f} of its limit, {bad} rows"


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
        check(feed_all(eng, "s", toks, cuts), want, dtype, f"{case} {cuts}", noise(case, toks))
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
        check(torch.cat(got[i]), oracle(case, seqs[i]), dtype, f"sequence {i}", noise(case, seqs[i]))
    assert eng.kv.used_blocks == 0


@pytest.mark.parametrize("dev,dtype", EXACT)
def test_long_decoding_keeps_the_state(dev, dtype):
    """300 single tokens with recurrences that forget slowly, chunks passed several times."""
    cfg = config([mamba(), delta(), parallel(chunk=40)], width=32, vocab=90)
    w = weights(cfg, seed=3)
    w["l0.mix.dt_bias"] -= 3
    w["l1.mix.dt_bias"] -= 3
    w["l2.mix.right.a2.b"] += 4
    toks = tokens(cfg, 330)
    want = oracle("slow", toks, cfg, w)
    eng = engine(None, dev, dtype, cfg=cfg, w=w)
    check(feed_all(eng, 0, toks, [30] + [1] * 300), want, dtype)


@pytest.mark.parametrize("dev,dtype", EXACT)
@pytest.mark.parametrize("chunk", [63, 64, 65])
@pytest.mark.parametrize("decode", [False, True])
def test_the_chunks_edge_shows(dev, dtype, chunk, decode):
    """One token's key stands out in an attention layer: positions that still see it and the first that does not, in a prompt and in
    decoding, at block borders.  (The oracle itself is shown to be sensitive to a chunk that is one off.)"""
    cfg = config([parallel(chunk=chunk, heads=2, kv_heads=1, dim=16, vdim=20, rot=2, scaling=None, base=1e9, softcap=20.0, scale=1.0, left=1.0, right=0.05)],
                 width=32, vocab=60, ff=None)
    w = weights(cfg, seed=5)
    w["embed"][:, 5] = 1.0                                           # every query has this
    w["embed"][7] = 0
    w["embed"][7, 3] = 3.0                                           # token 7's key is along one direction every query likes
    p = "l0.mix.left."
    w[p + "q"] *= 0.1
    w[p + "q"][:, 5] = 2.0
    w[p + "k"] *= 0.1
    w[p + "k"][:, 3] = 2.0
    w[p + "q.norm"][:], w[p + "k.norm"][:] = 1.0, 1.0
    w[p + "v"][:, 3] = 2.0
    toks = [t if t != 7 else 8 for t in tokens(cfg, 3 * chunk, seed=2)]
    toks[chunk - 1] = toks[chunk + 3] = 7
    want = oracle(("edge", chunk), toks, cfg, w)
    off = json.loads(json.dumps(cfg))
    off["layers"][0]["mixer"]["left"]["mask"]["size"] = chunk + 1
    moved = (oracle(("edge+1", chunk), toks, off, w) - want).abs().amax(-1)
    assert moved[chunk] > 0.2 and moved[2 * chunk] > 0.2 and moved[:chunk].max() == 0
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
    assert registry.for_path(d).name == "Lugovik" and lugovik.load_config(d).to_config()["layers"] == cfg["layers"]
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
    na, nb = noise(case, toks["a"]), noise(case, toks["b"])
    check(got, torch.stack([la[0], la[69], la[70], lb[2], la[79]]), dtype, off=torch.stack([na[0], na[69], na[70], nb[2], na[79]]))
    assert not (out / "2.f32").exists()


def test_configuration_and_checkpoint_errors(tmp_path):
    cfg, w = CASES["mixed"], weights(CASES["mixed"])
    load = lugovik.LugovikHParams.from_config
    mix = lambda c, i: c["layers"][i]["mixer"]                       # noqa: E731
    for edit in (lambda c: mix(c, 0)["left"].update(heads=7), lambda c: mix(c, 0)["left"]["rot"].update(dims=7), lambda c: mix(c, 0)["left"]["rot"].update(dims=26),
                 lambda c: mix(c, 1).update(groups=4), lambda c: mix(c, 1).update(norm_groups=7), lambda c: mix(c, 2).update(kv_heads=3),
                 lambda c: mix(c, 2).update(conv=0), lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="moe"),
                 lambda c: c.update(architecture="Other")):
        c = json.loads(json.dumps(cfg))
        edit(c)
        with pytest.raises(ValueError):
            load(c)
    hp = load(cfg)
    short = dict(list(w.items())[:-1])
    with pytest.raises(KeyError):
        list(lugovik.iter_checkpoint(write_model(tmp_path / "a", cfg, short), hp))
    with pytest.raises(ValueError):
        list(lugovik.iter_checkpoint(write_model(tmp_path / "b", cfg, dict(w, extra=w["head"])), hp))
    with pytest.raises(ValueError):
        list(lugovik.iter_checkpoint(write_model(tmp_path / "c", cfg, dict(w, head=w["head"][:-1])), hp))
    assert len(list(lugovik.iter_checkpoint(write_model(tmp_path / "e", cfg, dict(w, **{"l2.norm2": w["l1.norm2"]})), hp))) == len(w)     # a norm without its sublayer
    with pytest.raises(ValueError):
        lugovik.LugovikModel(hp, dict(w, **{"l2.mix.a1": w["l2.mix.a1"][:-1]}).items())
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
    assert registry.preset("lugovik-tiny").n_layer == 4 and registry.preset("lugovik-lite").n_params() > 5e8


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
@pytest.mark.parametrize("chunk", [64, 100, 512])
def test_tensor_core_shapes_in_the_model(chunk):
    """Head sizes of the tensor-core kernels: whole prompts, portions, short portions, decoding; two sequences at once."""
    cfg = config([mamba(heads=4, vdim=64, state=128, conv=4), delta(heads=3, kv_heads=3, dim=128, vdim=128),
                  parallel(heads=4, kv_heads=2, dim=128, vdim=128, rot=128, chunk=chunk, scale=128 ** -0.5, rheads=2, rdim=128, rvdim=128),
                  delta(heads=4, kv_heads=2, dim=64, vdim=64), mamba(heads=4, vdim=64, state=64, groups=2, norm_groups=2)], width=256, vocab=500, ff=512)
    w = weights(cfg, seed=1, rank=32)
    toks = tokens(cfg, 330)
    want = oracle(("wide", chunk), toks, cfg, w)
    eng = engine(None, "cuda", BF16, cfg=cfg, w=w)
    for cuts in ([330], [200, 70, 60], [100, 9, 2, 30], [65, 129, 63], [290] + [1] * 40):
        check(feed_all(eng, 0, toks, cuts), want, BF16, f"{cuts}", noise(("wide", chunk), toks, cfg, w))
        eng.end_feed(0)
    other = tokens(cfg, 290, seed=9)
    wo = oracle(("wide-b", chunk), other, cfg, w)
    got = {0: [], 1: []}
    for (a0, a1), (b0, b1) in zip(((0, 140), (140, 141), (141, 330)), ((0, 70), (70, 200), (200, 290))):
        out = eng.feed([(0, toks[a0:a1], range(a1 - a0)), (1, other[b0:b1], range(b1 - b0))])
        got[0].append(out[:a1 - a0])
        got[1].append(out[a1 - a0:])
    check(torch.cat(got[0]), want, BF16, off=noise(("wide", chunk), toks, cfg, w))
    check(torch.cat(got[1]), wo, BF16, off=noise(("wide-b", chunk), other, cfg, w))
    ops.nat().check_status()
