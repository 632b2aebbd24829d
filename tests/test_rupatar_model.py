"""Rupatar through the engine -- scheduler, paged and pooled rows, state slots, graphs -- against the plain oracle on whole sequences."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import rupatar_oracle as O
from jittorinfer_b200 import ops
from jittorinfer_b200.models import registry, rupatar
from jittorinfer_b200.runtime.engine import EngineConfig, LLMEngine
from jittorinfer_b200.runtime.sampling import SamplingParams
from rupatar_cases import CASES, attention, config, hgrn2, mlstm, moe, tokens, weights, write_model

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
    """How far the logits of each position move when every weight is off by about one bf16 rounding (a few draws, the largest): what a bf16
    run may differ by."""
    key = (case, tuple(toks), "noise")
    if key not in _oracle:
        cfg = cfg or CASES[case]
        offs = []
        for seed in range(3):
            g = torch.Generator().manual_seed(seed)
            moved = {k: t * (1 + 2.0 ** -8 * torch.randn(t.shape, generator=g)) for k, t in (w or weights(cfg)).items()}
            with torch.no_grad():
                offs.append(rows_off(O.forward(cfg, moved, toks), oracle(case, toks, cfg, w)))
        _oracle[key] = torch.stack(offs).amax(0)
    return _oracle[key]


def rows_off(got, want):
    """Per row: centred difference over the vocabulary against the size of the logits."""
    d = (got - want).double()
    return (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().std()


def engine(case, dev, dtype, n_ctx=1024, n_parallel=4, cfg=None, w=None, **kw):
    cfg = cfg or CASES[case]
    hp = rupatar.RupatarHParams.from_config(cfg)
    m = rupatar.RupatarModel(hp, (w or weights(cfg)).items(), dtype=dtype, device=dev, max_positions=n_ctx)
    kw.setdefault("n_batch", n_ctx)
    kw.setdefault("graph_buckets", (1, 2, 4))
    return LLMEngine(m, EngineConfig(n_ctx=n_ctx, n_parallel=n_parallel, n_ctx_slot=kw.pop("n_ctx_slot", n_ctx), **kw))


def check(got, want, dtype, what="", off=None):
    """``off``: what rounding may do (``noise``), for bf16.  A token whose experts are a close call may be further off."""
    err = rows_off(got, want)
    if dtype == F32:
        assert err.max() < 1e-4, f"{what}: row {int(err.argmax())} is off by {err.max():.2e}"
    else:
        lim = 0.03 + 3 * off
        bad = int((err > lim).sum())
        assert bad <= max(1, len(err) // 10) and err.median() < 0.05, f"{what}: median {err.median():.3f}, worst {(err / lim).max():.3f} of its limit, {bad} rows of {len(err)}"


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
        check(feed_all(eng, "s", toks, cuts), want, dtype, f"{case} {cuts}", noise(case, toks) if dtype == BF16 else None)
        eng.end_feed("s")
    assert eng.kv.used_blocks == 0 and eng.kv.check()
    if dev == "cuda":
        assert eng.stats["graph_steps"] >= 150
        ops.nat().check_status()


@pytest.mark.parametrize("dev,dtype", EXACT)
@pytest.mark.parametrize("case", list(CASES))
def test_the_residual_after_every_layer(case, dev, dtype):
    toks, want, got = tokens(CASES[case], 40), [], []
    with torch.no_grad():
        O.forward(CASES[case], weights(CASES[case]), toks, want)
    eng = engine(case, dev, dtype)
    eng.model.tensor_hook = lambda name, t: got.append(t.cpu()) if name.endswith("ffn_out") else None
    eng.feed([(0, toks, [])])
    assert len(got) == len(want) == len(CASES[case]["layers"]) == len(eng.kv_cache)
    for r, (a, b) in enumerate(zip(got, want)):
        assert (a - b).abs().max() < 2e-4 * b.abs().max(), f"layer {r}"


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
        check(torch.cat(got[i]), oracle(case, seqs[i]), dtype, f"sequence {i}", noise(case, seqs[i]) if dtype == BF16 else None)
    assert eng.kv.used_blocks == 0


@pytest.mark.parametrize("dev,dtype", EXACT)
def test_long_decoding_keeps_the_state(dev, dtype):
    """300 single tokens with recurrences that forget slowly and blocks pooled one token at a time."""
    cfg = config([attention(size=30, pool=8, mlp=moe(experts=4, top=2)), hgrn2(), mlstm(mlp=moe(shared=None))], width=32, groups=2, vocab=90)
    w = weights(cfg, seed=3)
    w["l1.mix.f.b"] += 3
    w["l2.mix.f.b"] += 3
    toks = tokens(cfg, 330)
    want = oracle("slow", toks, cfg, w)
    eng = engine(None, dev, dtype, cfg=cfg, w=w)
    check(feed_all(eng, 0, toks, [30] + [1] * 300), want, dtype)


def far_case(where):
    """One token stands out: attention finds its key -- alone in a wide window, or as a part of a pooled block -- or a recurrence writes its mark
    into a state that hardly fades; everything else is small.  (An attention layer before it makes the marked one mix values.)"""
    marked = {"window": attention(heads=2, kv_heads=1, dim=16, vdim=20, rot=2, base=1e9, scale=0.7, size=400, pool=4),
              "pool": attention(heads=2, kv_heads=1, dim=16, vdim=20, rot=2, base=1e9, scale=1.6, size=20, pool=4), "hgrn2": hgrn2(), "mlstm": mlstm(gate_cap=15.0)}[where]
    cfg = config([attention(vdim=10, kv_heads=2, size=9), marked, attention(vdim=10, kv_heads=2, size=9, v_mix=False)], width=32, groups=2, vocab=60)
    w = weights(cfg, seed=5)
    w["embed"][:, 5] = 1.0                                           # every query has this
    w["embed"][:, 3] = 0
    w["embed"][7] = 0
    w["embed"][7, 3] = 3.0
    for i in (0, 2):
        w[f"l{i}.mix.o"] *= 0.1
        w[f"l{i}.mix.o.b"] *= 0.1
    p = "l1.mix."
    if marked["type"] == "attention":                                # token 7's key is along one direction every query likes
        for k in ("q", "k", "q.b", "k.b"):
            w[p + k] *= 0.02
        w[p + "q"][15::16, 5], w[p + "k"][15, 3], w[p + "v"][:, 3], w[p + "k"][3, 5], w[p + "vmix"] = 2.0, 2.0, 4.0, 2.0, torch.tensor(0.25)
    elif where == "hgrn2":                                           # its channels are written by that token only
        w[p + "f"] *= 0.2
        w[p + "f"][:, 3], w[p + "f.b"][:], w[p + "lower"][:], w[p + "v"][:, 3] = -6.0, 7.0, 0.0, 4.0
    else:                                                            # or it opens the input gates
        w[p + "i"][:, 3], w[p + "i.b"][:], w[p + "f.b"][:], w[p + "v"][:, 3] = 3.0, -1.0, 8.0, 4.0
        w[p + "q"][:, 5], w[p + "k"][:, 3], w[p + "k"][:, 5] = 2.0, 2.0, 2.0          # q . k well away from 0
    return cfg, w


@pytest.mark.parametrize("dev,dtype", EXACT)
@pytest.mark.parametrize("where", ["window", "pool", "hgrn2", "mlstm"])
def test_a_token_far_back_shows(where, dev, dtype):
    """Prompts, portions and decoding; the oracle itself is shown to be sensitive to the token."""
    cfg, w = far_case(where)
    plain = [t if t != 7 else 8 for t in tokens(cfg, 260, seed=2)]
    for place in (0, 63, 64, 130):
        toks = list(plain)
        toks[place] = 7
        want = oracle((where, place), toks, cfg, w)
        shift = (oracle((where, "plain"), plain, cfg, w) - want).abs().amax(-1)
        assert shift[place + 100:].min() > 0.02 and (place == 0 or shift[:place].max() == 0), shift[place + 100:].min()
        eng = engine(None, dev, dtype, cfg=cfg, w=w)
        for cuts in ([260], [place + 1, 2], [180] + [1] * 80):
            check(feed_all(eng, 0, toks, cuts), want, dtype, f"{place} {cuts}")
            eng.end_feed(0)


@pytest.mark.parametrize("dev,dtype", EXACT)
@pytest.mark.parametrize("size,pool", [(63, 8), (64, 16), (65, 5), (20, 64)])
def test_a_token_at_the_windows_edge_and_in_its_block_shows(size, pool, dev, dtype):
    """The oracle moves while the token is in the window, not between the window and the end of its block's wait, and again from then on; the
    engine follows in prompts, portions and decoding, also where the last layer reads the blend of values."""
    cfg, w = far_case("pool")
    cfg["layers"][1]["mixer"]["mask"] = {"size": size, "pool": pool}
    cfg["layers"] = cfg["layers"][:2]
    cfg["layers"][0]["mixer"]["mask"] = {"size": 1, "pool": 999}
    w = {k: t for k, t in w.items() if not k.startswith("l2.")}
    n = size + 2 * pool + 12
    plain = [t if t != 7 else 8 for t in tokens(cfg, n, seed=6)]
    for place in (0, pool - 1, pool):
        toks = list(plain)
        toks[place] = 7
        want = oracle(("edge", size, pool, place), toks, cfg, w)
        shift = (oracle(("edge", size, pool), plain, cfg, w) - want).abs().amax(-1)
        back = size + place // pool * pool + pool - 1                # the first position that sees its block
        assert shift[place:place + size].min() > 1e-2 and shift[back:].min() > 1e-3 and (place + size >= back or shift[place + size:back].max() == 0)
        eng = engine(None, dev, dtype, cfg=cfg, w=w)
        for cuts in ([n], [place + size, 1, 1, 2], [size] + [1] * (n - size), [back, 1, 3]):
            check(feed_all(eng, 0, toks, cuts), want, dtype, f"{place} {cuts}")
            eng.end_feed(0)


@pytest.mark.parametrize("dev,dtype", EXACT)
def test_every_part_of_the_model_shows(dev, dtype):
    """A change of any one tensor's weights moves the oracle's logits, and the engine's with them."""
    cfg = CASES["mixed"]
    toks, base = tokens(cfg, 12, seed=4), weights(cfg)
    names = [n for n in base if not n.startswith("l") or n.startswith(("l1.", "l2.", "l3.")) and ".e" not in n] + ["l0.mix.v", "l4.mix.vmix", "l6.mix.vmix", "l1.mlp.e0.up", "l4.mlp.e3.down"]
    for n in names:
        w = dict(base, **{n: base[n] * 1.5 + (0.1 if "lower" not in n else -0.02)})
        with torch.no_grad():
            want = O.forward(cfg, w, toks)
        if ".mlp.e" not in n and n not in ("l2.mix.vmix", "embed"):   # l2 is the first that mixes: its own blend is not used
            assert rows_off(want, oracle("mixed", toks)).max() > 1e-3, n
        check(feed_all(engine(None, dev, dtype, cfg=cfg, w=w, n_ctx=64, cuda_graphs=False), 0, toks, [8, 1]), want, dtype, n)


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
    """A prompt that extends everything a slot holds continues from its state; one that shares only a part of it is evaluated from the
    start, because the state exists at the end only."""
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
    _, n = run(first + out[:5] + tokens(cfg, 12, seed=8))
    assert n == 12 + 5                                               # continued from the state
    _, n = run(first)                                                # a proper prefix of what the slot holds
    assert n == 95


def test_sampling_modes_cancel_reset_and_poisoned_blocks(monkeypatch):
    monkeypatch.setenv("JITTORINFER_KV_POISON", "1")                 # freed blocks of every layer, pooled ones too, are filled with NaN
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


# ---- files, registry, command lines -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
def test_folder_model_through_the_registry_and_the_trace_runner(tmp_path, dev, dtype):
    case = "mixed"
    cfg, w = CASES[case], weights(CASES[case])
    d = write_model(tmp_path / "m", cfg, w)
    hp = rupatar.load_config(d)
    assert registry.for_path(d).name == "Rupatar" and rupatar.RupatarHParams.from_config(hp.to_config()) == hp
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
    la, lb, na, nb = oracle(case, toks["a"]), oracle(case, toks["b"]), noise(case, toks["a"]), noise(case, toks["b"])
    got = torch.cat([read(0), read(1), read(3)])
    check(got, torch.stack([la[0], la[69], la[70], lb[2], la[79]]), dtype, off=torch.stack([na[0], na[69], na[70], nb[2], na[79]]))
    assert not (out / "2.f32").exists()


def test_configuration_and_checkpoint_errors(tmp_path):
    cfg, w = CASES["mixed"], weights(CASES["mixed"])
    load = rupatar.RupatarHParams.from_config
    mix = lambda c, i: c["layers"][i]["mixer"]                       # noqa: E731
    mlp = lambda c, i: c["layers"][i]["mlp"]                         # noqa: E731
    for edit in (lambda c: mix(c, 0).update(heads=7), lambda c: mix(c, 0)["rot"].update(dims=7), lambda c: mix(c, 0)["rot"].update(dims=26), lambda c: mix(c, 2)["mask"].update(size=0),
                 lambda c: mix(c, 0)["mask"].update(pool=-1), lambda c: mix(c, 1).update(heads=0), lambda c: mix(c, 4).update(vdim=41), lambda c: c["layers"][0].update(type="other"),
                 lambda c: mlp(c, 0).update(kind="other"), lambda c: mlp(c, 1)["router"].update(top=9), lambda c: mlp(c, 2)["router"].update(experts=300), lambda c: c["norm"].update(groups=7),
                 lambda c: c["norm"].update(groups=0), lambda c: c.update(architecture="Other")):
        c = json.loads(json.dumps(cfg))
        edit(c)
        with pytest.raises(ValueError):
            load(c)
    hp = load(cfg)
    assert hp.first_mix == 2 and load(CASES["states"]).first_mix == -1
    with pytest.raises(KeyError):
        list(rupatar.iter_checkpoint(write_model(tmp_path / "a", cfg, dict(list(w.items())[:-1])), hp))
    with pytest.raises(ValueError):
        list(rupatar.iter_checkpoint(write_model(tmp_path / "b", cfg, dict(w, extra=w["head"])), hp))
    with pytest.raises(ValueError):
        list(rupatar.iter_checkpoint(write_model(tmp_path / "c", cfg, dict(w, head=w["head"][:-1])), hp))
    assert len(list(rupatar.iter_checkpoint(write_model(tmp_path / "e", cfg, dict(w, **{"l3.norm2": w["l1.norm2"], "l0.mix.vmix": w["l2.mix.vmix"]})), hp))) == len(w)     # a norm without its sublayer, an unused blend
    with pytest.raises(ValueError):
        rupatar.RupatarModel(hp, list(w.items())[:-1])
    with pytest.raises(KeyError):
        rupatar.RupatarModel(hp, [("l0.mlp.e99.up", w["l0.mlp.e0.up"])])
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
    assert registry.preset("rupatar-tiny").n_layer == 4 and registry.preset("rupatar-lite").n_params() > 4e9


@pytest.mark.parametrize("dev,dtype", EXACT)
def test_defragmentation_moves_rows_and_pooled_rows(dev, dtype):
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
def test_tensor_core_shapes_in_the_model():
    """Sizes of the tensor-core kernels: whole prompts, portions, short portions, decoding; two sequences at once."""
    cfg = config([attention(heads=4, kv_heads=2, dim=128, vdim=128, rot=64, scale=128 ** -0.5, size=100, pool=16, mlp=moe(ff=128, experts=16, top=4, shared=256)), hgrn2(heads=2, dim=128, vdim=128),
                  attention(heads=4, kv_heads=1, dim=64, vdim=64, rot=64, scale=0.125, size=64, pool=8, v_mix=False, mlp=moe(ff=128, experts=8, top=2, shared=192)),
                  mlstm(heads=2, dim=128, vdim=128, mlp=moe(ff=128, shared=128)), hgrn2(heads=4, dim=64, vdim=64),
                  attention(heads=2, kv_heads=2, dim=128, vdim=128, rot=128, scale=128 ** -0.5, size=33, pool=5), mlstm(heads=4, dim=64, vdim=64)],
                 width=256, vocab=500, groups=8)
    w = weights(cfg, seed=1)
    toks, other = tokens(cfg, 330), tokens(cfg, 290, seed=9)
    want, wo = oracle("wide", toks, cfg, w), oracle("wide", other, cfg, w)
    lim, lo = noise("wide", toks, cfg, w), noise("wide", other, cfg, w)
    eng = engine(None, "cuda", BF16, cfg=cfg, w=w)
    for cuts in ([330], [200, 70, 60], [100, 9, 2, 30], [65, 129, 63], [290] + [1] * 40):
        check(feed_all(eng, 0, toks, cuts), want, BF16, f"{cuts}", lim)
        eng.end_feed(0)
    got = {0: [], 1: []}
    for (a0, a1), (b0, b1) in zip(((0, 140), (140, 141), (141, 330)), ((0, 70), (70, 200), (200, 290))):
        out = eng.feed([(0, toks[a0:a1], range(a1 - a0)), (1, other[b0:b1], range(b1 - b0))])
        got[0].append(out[:a1 - a0])
        got[1].append(out[a1 - a0:])
    check(torch.cat(got[0]), want, BF16, off=lim)
    check(torch.cat(got[1]), wo, BF16, off=lo)
    assert ops.nat().launches_by_name.get("gqa_prefill", 0) > 0 and ops.nat().launches_by_name.get("state_chunk", 0) > 0
    ops.nat().check_status()
