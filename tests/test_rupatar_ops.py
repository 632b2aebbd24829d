"""Each mechanism of the Rupatar layers alone, against the plain oracle: the product's ops on the CPU and its kernels on a GPU."""
import math

import pytest
import torch

import rupatar_oracle as O
from jittorinfer_b200 import ops
from jittorinfer_b200.models import folder
from jittorinfer_b200.ops.specs import Gqa, RowNorms, StateMix

GPU = pytest.mark.gpu
WHERE = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda", torch.float32, id="cuda-f32", marks=GPU),
         pytest.param("cuda", torch.bfloat16, id="cuda-bf16", marks=GPU)]
F32, BF16 = torch.float32, torch.bfloat16


def tol(dtype):
    return 3e-5 if dtype == F32 else 2.5e-2


def close(a, b, dtype, what="", scale=1.0):
    a, b = a.double().cpu(), b.double().cpu()
    err = (a - b).abs().max().item()
    assert err <= scale * tol(dtype) * max(1.0, b.abs().max().item()), f"{what}: {err} of {b.abs().max().item()}"


def rnd(*shape, seed=0, scale=1.0, mean=0.0):
    return (mean + torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * scale).bfloat16().float()


def i32(x, dev="cpu"):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def starts(q_lens, dev):
    return i32([0] + torch.tensor(q_lens).cumsum(0).tolist(), dev)


def moved(spec, dev):
    return type(spec)(**{k: v.to(dev) if isinstance(v, torch.Tensor) else v for k, v in vars(spec).items()})


# ---- recurrences ---------------------------------------------------------------------------------------------------------------
def run_state(kind, dev, dtype, H, K, V, cuts, lens, seed=0, forget=0.0, write=0.0, cap=6.0, lower=0.4, mark=None, single_ok=True, off=(8, 16)):
    """Sequences interleaved in portions, alone and together, against the oracle on whole ones; slots hold what earlier sequences left.
    ``forget``, ``write``: added to the gates' pre-activations; ``mark`` = (token, factor): values that stand out."""
    q_off, v_off = off[0], off[0] + 2 * H * K + off[1]                # columns between the parts belong to nobody
    cols = v_off + H * V
    dec_w = H * K if kind == "hgrn" else 2 * H
    m = StateMix(kind, H, K, V, q_off=q_off, k_off=q_off + H * K, v_off=v_off, eps=1e-2, out_scale=1.3)
    if kind == "hgrn":
        m.bias, m.lower, m.norm_w = rnd(H * K, seed=seed + 1) + forget, torch.rand(H * K, generator=torch.Generator().manual_seed(seed)) * lower, rnd(V, seed=seed + 3, scale=0.2, mean=1.0)
        m.lower[::2] = 0
    else:
        m.norm_w, m.q_scale, m.gate_cap = rnd(H * V, seed=seed + 3, scale=0.2, mean=1.0), K ** -0.5, cap
        m.bias = torch.tensor([write + 0.013 * h for h in range(H)] + [forget - 0.017 * h for h in range(H)])
    data, want = [], []
    for j, n in enumerate(lens):
        proj, gate = rnd(n, cols, seed=50 + 9 * j + seed), rnd(n, H * V, seed=51 + 9 * j + seed)
        dec = rnd(n, dec_w, seed=52 + 9 * j + seed, scale=1.5)
        if mark is not None and mark[0] < n:
            proj[mark[0], v_off:] *= mark[1]
        data.append((proj, dec, gate))
        p, z = proj.double(), dec.double()
        part = lambda o, w: p[:, o:o + H * w].view(n, H, w)          # noqa: B023,E731
        if kind == "hgrn":
            f = m.lower.double() + (1 - m.lower.double()) * O.sigmoid(z + m.bias.double())
            q = part(q_off, K)
            o, S = O.hgrn2_scan(q * O.sigmoid(q), f.view(n, H, K), part(v_off, V))
            want.append((1.3 * (O.rms(o, m.eps) * m.norm_w.double()).reshape(n, -1), (S,)))
        else:
            z = z + m.bias.double()
            i, f = cap * torch.tanh(z[:, :H] / cap), O.log_sigmoid(cap * torch.tanh(z[:, H:] / cap))
            o, S = O.mlstm_scan(part(q_off, K) * K ** -0.5, part(q_off + H * K, K), part(v_off, V), i, f)
            want.append((1.3 * O.rms(o, m.eps).reshape(n, -1) * m.norm_w.double() * O.sigmoid(gate.double()), S))
    md = moved(m, dev)
    state, extra = torch.full((4, H, K, V), 3.0, device=dev), torch.full((4, H, K + 1), 3.0, device=dev) if kind == "mlstm" else None
    at, slots = [0] * len(lens), (3, 1)
    chunks = ops.nat().launches_by_name.get("state_chunk", 0) if dev == "cuda" else 0
    for cut in cuts:
        part = [(j, at[j], n) for j, n in enumerate(cut) if n]
        proj, dec, gate = (torch.cat([data[j][k][p:p + n] for j, p, n in part]).to(dev) for k in range(3))
        proj, dec, gate = proj.to(dtype), dec.to(dtype), gate.to(dtype)
        out = torch.full((proj.shape[0], H * V + 8), 9.0, dtype=dtype, device=dev)
        single = single_ok and all(n == 1 for *_, n in part)
        ops.state_mix(md, proj, dec, None if kind == "hgrn" else gate, None, state, i32([slots[j] for j, *_ in part], dev),
                      i32([p + k for _, p, n in part for k in range(n)], dev), starts([n for *_, n in part], dev), single, out[:, :H * V], extra)
        close(out[:, :H * V], torch.cat([want[j][0][p:p + n] for j, p, n in part]), dtype, f"cut {cut} at {at}")
        assert bool((out[:, H * V:] == 9).all())
        for j, _, n in part:
            at[j] += n
    assert tuple(at) == tuple(lens)
    for j in range(len(lens)):
        close(state[slots[j]], want[j][1][0], dtype, "state")
        if kind == "mlstm":
            close(extra[slots[j], :, :K], want[j][1][1], dtype, "sum of keys")
            close(extra[slots[j], :, K], want[j][1][2], F32, "maximum")
    for t in (state, extra) if kind == "mlstm" else (state,):
        assert bool((t[0] == 3).all()) and bool((t[2] == 3).all())
    if dev == "cuda":                                                # portions of these sizes take the tensor cores
        many = any(max(c) > 1 for c in cuts) or not single_ok
        assert (ops.nat().launches_by_name.get("state_chunk", 0) > chunks) == (dtype == BF16 and many and K in (64, 128) and V % 16 == 0)
        ops.nat().check_status()


SIZES = [(1, 1, 1), (3, 5, 7), (2, 20, 24), (4, 33, 40), (2, 64, 64), (3, 64, 48), (2, 128, 128), (1, 128, 16), (1, 200, 72), (2, 96, 144)]


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("H,K,V", SIZES)
@pytest.mark.parametrize("kind", ["hgrn", "mlstm"])
def test_recurrence_in_portions_equals_one_pass(kind, H, K, V, dev, dtype):
    off = (0, 0) if (K, V) == (64, 48) else (8, 16)
    run_state(kind, dev, dtype, H, K, V, [(1, 3), (1, 1), (2, 0), (67, 4), (1, 1), (0, 1), (31, 50), (17, 1), (1, 0), (29, 0)], (150, 61), forget=1.0, off=off)
    run_state(kind, dev, dtype, H, K, V, [(150, 0), (0, 61)], (150, 61), seed=1, forget=2.0, off=off)
    run_state(kind, dev, dtype, H, K, V, [(1, 1)] * 3 + [(5, 5)], (8, 8), seed=2, single_ok=False, off=off)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("H,K,V", [(2, 20, 24), (1, 128, 32)])
@pytest.mark.parametrize("kind", ["hgrn", "mlstm"])
def test_recurrence_remembers_over_long_prompts_and_long_decoding(kind, H, K, V, dev, dtype):
    """Slow decays and one token that stands out: what it wrote is still there; a lost or doubled update would stay."""
    run_state(kind, dev, dtype, H, K, V, [(260, 0), (0, 1)] + [(1, 1)] * 60, (320, 61), forget=6.0, lower=0.0, mark=(2, 60.0))
    run_state(kind, dev, dtype, H, K, V, [(129, 300), (191, 20)], (320, 320), forget=6.0, mark=(33, 60.0))


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("H,K,V", [(2, 20, 24), (1, 64, 32), (1, 128, 32)])
@pytest.mark.parametrize("kind", ["hgrn", "mlstm"])
def test_recurrence_survives_very_fast_decays(kind, H, K, V, dev, dtype):
    """Decays down to zero: products over a few tokens underflow, their quotients must not matter."""
    run_state(kind, dev, dtype, H, K, V, [(140, 61), (10, 0)], (150, 61), forget=-30.0, lower=0.0, cap=20.0)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("H,K,V", [(2, 20, 24), (1, 64, 32)])
@pytest.mark.parametrize("write,forget,cap", [(-8.0, 3.0, 30.0), (14.0, 3.0, 30.0), (-3.0, -2.0, 30.0), (0.0, 40.0, 1.0), (3.0, 0.0, 0.5)])
def test_mlstm_gates_in_every_regime(write, forget, cap, H, K, V, dev, dtype):
    """A maximum that stays at what the forget gates leave of its start, one that follows the input gates, states so small that the output's
    divisor is exp(-m), and gates at their cap."""
    run_state("mlstm", dev, dtype, H, K, V, [(1, 40), (70, 1), (1, 1), (1, 1), (47, 18)], (120, 61), write=write, forget=forget, cap=cap)


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_mlstm_maximum_over_thousands_of_tokens(dev, dtype):
    """More tokens than one pass of the gates' scan holds; the maximum of the last is carried on."""
    run_state("mlstm", dev, dtype, 1, 4, 4, [(2500, 3), (1, 1), (2, 2)], (2503, 6), write=-2.0, forget=5.0, cap=9.0)


@GPU
@pytest.mark.parametrize("kind", ["hgrn", "mlstm"])
def test_recurrence_keeps_a_mark_among_a_thousand_tokens(kind):
    run_state(kind, "cuda", F32, 1, 16, 16, [(700, 0)] + [(1, 0)] * 400 + [(0, 1)], (1100, 1), forget=9.0, lower=0.0, cap=30.0, mark=(3, 300.0))
    run_state(kind, "cuda", BF16, 1, 128, 16, [(1000, 0), (100, 1)], (1100, 1), forget=9.0, lower=0.0, cap=30.0, mark=(3, 300.0))


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("K", [16, 64])
@pytest.mark.parametrize("kind", ["hgrn", "mlstm"])
def test_padding_rows_leave_every_state_alone(kind, K, dev, dtype):
    H, V = 2, 16
    m = moved(StateMix(kind, H, K, V, q_off=0, k_off=H * K, v_off=2 * H * K, bias=rnd(H * K if kind == "hgrn" else 2 * H), lower=torch.zeros(H * K), norm_w=rnd(V if kind == "hgrn" else H * V), gate_cap=5.0), dev)
    st, ex = torch.full((2, H, K, V), 5.0, device=dev), torch.full((2, H, K + 1), 5.0, device=dev)
    for single in (True, False):
        out = torch.empty(2, H * V, dtype=dtype, device=dev)
        dec = rnd(2, H * K if kind == "hgrn" else 2 * H).to(dev, dtype)
        ops.state_mix(m, rnd(2, 2 * H * K + H * V).to(dev, dtype), dec, rnd(2, H * V).to(dev, dtype) if kind == "mlstm" else None, None, st, i32([-1, -1], dev), i32([0, 9], dev),
                      i32([0, 1, 2], dev), single, out, ex if kind == "mlstm" else None)
    assert bool((st == 5).all()) and bool((ex == 5).all())


# ---- attention -----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("stretch", [1.0, 2.0, 7.5])
@pytest.mark.parametrize("dims", [2, 12, 64])
def test_rotation_table_is_stretched(dims, stretch):
    t = folder.rope_table(300, folder.Rotation(dims, 700.0, stretch=stretch), "cpu")
    v = torch.zeros(300, 1, dims, dtype=torch.float64)
    v[..., ::2] = 1
    r = O.rotate(v, dict(dims=dims, base=700.0, scaling=dict(factor=stretch)))[:, 0]
    assert (t[..., 0] - r[:, ::2]).abs().max() < 1e-6 and (t[..., 1] - r[:, 1::2]).abs().max() < 1e-6


class Paged:
    """Sequences over shuffled blocks of one cache whose other rows, and all pooled rows, are NaN."""

    def __init__(self, m, lens, dtype, dev, bs=64):
        nb = [(n + bs - 1) // bs for n in lens]
        perm = torch.randperm(sum(nb) + 2, generator=torch.Generator().manual_seed(3)).tolist()
        nan = lambda n: torch.full((n, m.kv_row), float("nan"), dtype=dtype, device=dev)          # noqa: E731
        self.cache, self.pool = nan((sum(nb) + 2) * bs), nan((sum(nb) + 2) * m.pool_rows(bs))
        self.tables, self.bs = torch.zeros(len(lens), max(nb), dtype=torch.int32), bs
        for j, n in enumerate(nb):
            for i in range(n):
                self.tables[j, i] = perm.pop()

    def slots(self, j, pos):
        return [int(self.tables[j, p // self.bs]) * self.bs + p % self.bs for p in pos]


def run_attention(m, dev, dtype, cuts, lens, rot, seed=0, hot=(), single_ok=True):
    """q, k, v through gqa_qkv_post and gqa_attention in portions, against the oracle on whole sequences.  ``hot``: (sequence, position) pairs
    whose keys every later query likes and whose values stand out."""
    H, G, D, V = m.heads, m.kv_heads, m.dim, m.vdim
    widths = (H * D, G * D, G * V, H * V, G * V)                     # q, k, v, gate, the first layer's values
    seqs = [[rnd(n, c, seed=30 + seed + 7 * j + i) for i, c in enumerate(widths)] for j, n in enumerate(lens)]
    for s in seqs if hot else ():                                    # along the unrotated last dimension
        s[0].view(-1, H, D)[..., -1] = 6.0 * D ** 0.5
        s[1].view(-1, G, D)[..., -1] = 0
    for j, p in hot:
        seqs[j][1].view(-1, G, D)[p] = 0
        seqs[j][1].view(-1, G, D)[p, :, -1] = 9.0
        seqs[j][2][p] = 5.0 + p % 7
        seqs[j][4][p] = 5.0 + p % 7
    want = []
    for q, k, v, g, v0 in ([t.double() for t in s] for s in seqs):
        n = q.shape[0]
        q, k = (O.rms(O.rotate(x.view(n, -1, D), rot), m.eps) for x in (q, k))
        if m.v_mix is not None:
            v = O.mix_values(v, v0, m.v_mix)
        want.append(O.attend(q, k, v.view(n, G, V), m.scale, m.window, m.pool).reshape(n, H * V) * O.sigmoid(g))
    pg = Paged(m, lens, dtype, dev)
    table = folder.rope_table(max(lens), folder.Rotation(rot["dims"], rot["base"], stretch=rot["scaling"]["factor"]), dev)
    at, got, bounds = [0] * len(lens), [[] for _ in lens], torch.tensor((0,) + widths).cumsum(0).tolist()
    prefills = ops.nat().launches_by_name.get("gqa_prefill", 0) if dev == "cuda" else 0
    for cut in cuts:
        part = [(j, at[j], n) for j, n in enumerate(cut) if n]
        proj = torch.cat([torch.cat([x[p:p + n] for x in seqs[j]], 1) for j, p, n in part]).to(dev, dtype)
        q, k, v, g, v0 = (proj[:, a:b] for a, b in zip(bounds, bounds[1:]))
        pos = i32([p + i for _, p, n in part for i in range(n)], dev)
        slots = i32([s for j, p, n in part for s in pg.slots(j, range(p, p + n))], dev)
        q_lens, s_lens = [n for *_, n in part], [p + n for _, p, n in part]
        tables, lens_d, qs = pg.tables[[j for j, *_ in part]].to(dev), i32(s_lens, dev), starts(q_lens, dev)
        single = single_ok and max(q_lens) == 1
        qo = ops.gqa_qkv_post(m, q, k, v, table, pos, slots, pg.cache, v0, (pg.pool, tables, lens_d, qs, 64, single) if m.pool else None)
        out = torch.full((proj.shape[0], H * V + 8), 9.0, dtype=dtype, device=dev)
        meta = {"q_lens": q_lens, "s_lens": s_lens, "n_q_tiles": sum((x + 127) // 128 for x in q_lens), "total_kv": sum(s_lens), "kv_decode": 0}
        ops.gqa_attention(m, qo, pg.cache, g, tables, lens_d, qs, 64, max(q_lens), meta, out[:, :H * V], pg.pool)
        assert bool((out[:, H * V:] == 9).all())
        i = 0
        for j, _, n in part:
            got[j].append(out[i:i + n, :H * V])
            at[j] += n
            i += n
    assert tuple(at) == tuple(lens)
    for j in range(len(lens)):
        close(torch.cat(got[j]), want[j], dtype, f"sequence {j}")
    if dev == "cuda":                                                # the tensor-core kernel ran where it should
        assert (ops.nat().launches_by_name.get("gqa_prefill", 0) > prefills) == (dtype == BF16 and D == V == 128 and max(map(sum, cuts)) >= 64)
        ops.nat().check_status()
    return want


def gqa(H=4, G=2, D=24, V=20, rot=16, window=50, pool=6, scale=0.25, v_mix=0.3):
    return Gqa(H, G, D, V, rot, scale, window=window, sink=True, eps=1e-4, neighbours=True, unit=True, pool=pool, v_mix=v_mix, gate_each=True)


def rot(dims, base=900.0, factor=2.0):
    return dict(dims=dims, base=base, scaling=dict(factor=factor))


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("shape", [dict(), dict(H=1, G=1, D=2, V=1, rot=2, window=1, pool=1), dict(H=21, G=1, D=13, V=9, rot=6, window=37, pool=5), dict(H=6, G=6, D=64, V=64, rot=64, window=64, pool=64),
                                   dict(H=3, G=3, D=40, V=200, rot=20, window=1000, pool=3, v_mix=None), dict(H=34, G=2, D=32, V=36, rot=0, window=11, pool=75), dict(H=2, G=1, D=260, V=300, rot=64, window=20, pool=1),
                                   dict(H=4, G=2, D=128, V=128, rot=128, window=30, pool=2), dict(H=6, G=2, D=128, V=128, rot=64, window=100, pool=16), dict(H=2, G=1, D=32, V=16, rot=8, window=9, pool=0)])
def test_attention_in_portions_equals_one_pass(shape, dev, dtype):
    m = gqa(**shape)
    run_attention(m, dev, dtype, [(1, 2), (1, 1), (130, 3), (1, 1), (2, 60), (65, 33), (40, 0)], (240, 100), rot(m.rot))
    run_attention(m, dev, dtype, [(240, 0), (0, 100)], (240, 100), rot(m.rot, factor=1.0), seed=1)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("D", [24, 32, 128])
@pytest.mark.parametrize("window,pool", [(63, 8), (64, 16), (65, 7), (40, 64), (129, 4), (5, 100), (1, 1), (16, 3)])
def test_the_windows_edge_and_the_blocks_behind_it_show(window, pool, D, dev, dtype):
    """Keys that every query likes, at the ends of pooled blocks and cache blocks: seen alone while in the window, not at all until their block
    lies before it, then as a part of its mean.  In prompts, in portions that end at the edges, and in decoding across them."""
    n = 190 + window
    hot = [(0, 0), (0, pool), (0, 63), (1, pool - 1), (1, 64), (1, 66 + pool)]
    m = gqa(H=2, G=1, D=D, V=D, rot=16, window=window, pool=pool, scale=12.0 / D)
    for cuts in ([(n, n)], [(window, pool)] + [(1, 1)] * 5 + [(pool, window)] + [(1, 1)] * 3, [(64, 66 + pool)] + [(1, 1)] * 9 + [(window + 1, 1)] + [(1, 0)] * 5):
        left = [n - sum(c[j] for c in cuts) for j in (0, 1)]
        want = run_attention(m, dev, dtype, cuts + ([tuple(left)] if max(left) else []), (n, n), rot(16), hot=hot)
    seen = lambda i, j, h: j in O.seen_tokens(i, window) or j // pool in O.seen_blocks(i, window, pool)          # noqa: E731
    with_mark = [want[0][i].abs().max() for i in range(n) if seen(i, 0, 0) and i < pool]
    assert min(with_mark) > 0.5                                       # it does stand out


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_far_keys_among_many(dev, dtype):
    """One key a thousand tokens back: a single one in a wide window, or a part of a pooled block."""
    for D, window, pool in ((24, 2000, 8), (128, 2000, 8), (24, 30, 4), (128, 30, 4)):
        m = gqa(H=2, G=1, D=D, V=D, window=window, pool=pool, scale=(12.0 if window > 30 else 36.0) / D)
        run_attention(m, dev, dtype, [(1, 0), (1000, 0), (1, 0), (3, 0), (1, 0), (0, 1)], (1006, 1), rot(16), hot=[(0, 5)])


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_blocks_completed_by_single_tokens_and_by_portions_hold_the_same_means(dev, dtype):
    """Two tokens at a time, one at a time through either form of the step, all at once; blocks that reach over cache blocks."""
    for D, pool in ((24, 7), (32, 24)):
        m = gqa(D=D, V=D, window=10, pool=pool)
        for cuts, ok in (([(2, 2)] * 50, True), ([(1, 1)] * 100, True), ([(1, 1)] * 100, False), ([(100, 3), (0, 97)], True)):
            run_attention(m, dev, dtype, cuts, (100, 100), rot(16), single_ok=ok)


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_the_sink_shows(dev, dtype):
    """Scores far below and far above the sink's 0."""
    H, D, n = 2, 16, 70
    for sign in (-1.0, 1.0):
        q, v = torch.zeros(n, H * D), rnd(n, D, seed=3)
        q.view(n, H, D)[..., 0] = 1.0
        k = torch.zeros(n, D)
        k[:, 0] = sign
        m = Gqa(H, 1, D, D, 0, 0.4, window=20, sink=True, eps=1e-6, neighbours=True, unit=True, pool=5)
        o = O.attend(O.rms(q.double().view(n, H, D), 1e-6), O.rms(k.double().view(n, 1, D), 1e-6), v.double().view(n, 1, D), 0.4, 20, 5)
        assert (o.abs().max() < 0.2) == (sign < 0)
        pg = Paged(m, [n], dtype, dev)
        args = pg.tables.to(dev), i32([n], dev), i32([0, n], dev)
        parts = torch.cat([q, k, v], 1).to(dev, dtype).split([H * D, D, D], 1)
        qo = ops.gqa_qkv_post(m, *parts, torch.zeros(n, 0, 2, device=dev), i32(list(range(n)), dev),
                              i32(pg.slots(0, range(n)), dev), pg.cache, None, (pg.pool, *args, 64, False))
        out = torch.empty(n, H * D, dtype=dtype, device=dev)
        ops.gqa_attention(m, qo, pg.cache, None, *args, 64, n, None, out, pg.pool)
        close(out.view(n, H, D), o, dtype)


# ---- rows and products -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("d,groups", [(48, 1), (48, 3), (48, 6), (45, 9), (45, 45), (40, 8), (1024, 16), (2048, 8), (2560, 5), (5120, 8), (5120, 20), (8192, 2), (16384, 1024), (6144, 3)])
def test_norms_in_parts(d, groups, dev, dtype):
    T, E, k, eps = 5, 4, 3, 1e-2
    w, table = rnd(d, seed=1, scale=0.3, mean=1.0), rnd(20, d, seed=2)
    x, o, y, f = rnd(T, d, seed=3, scale=2.0), rnd(T, d, seed=4), rnd(T * k, d, seed=5), rnd(T, d, seed=6)
    for t in (table, x):                                             # parts of very different sizes
        t.copy_((t * (1 + torch.arange(groups)).repeat_interleave(d // groups) / groups).bfloat16())
    put, put32 = (lambda t: t.to(dev, dtype)), (lambda t: t.to(dev))          # noqa: E731
    nxt = RowNorms(eps, w.to(dev), groups=groups)
    norm = lambda v: O.group_norm(v.double(), w.double(), groups, eps)          # noqa: E731
    ids = i32([3, 0, 19, 7, 3], dev)
    rows, h, none = ops.embed_norm(put(table), ids, None, eps, nxt, 3.0)
    close(rows, 3.0 * table[ids.long().cpu()], F32)
    close(h, norm(3.0 * table[ids.long().cpu()]), dtype)
    assert none is None
    s, h, _ = ops.scaled_update(put32(x.clone()), put(o), None, nxt=nxt)
    close(s, x + o, F32)
    close(h, norm(x + o), dtype)
    dest = torch.randperm(T * k, generator=torch.Generator().manual_seed(7)).view(T, k).int()
    s, h, _ = ops.scaled_update(put32(x.clone()), None, None, moe=(put(y), dest.to(dev), None), dense=put(f), nxt=nxt)
    close(s, x + y[dest.long()].sum(1) + f, F32, scale=3)
    close(h, norm(x + y[dest.long()].sum(1) + f), dtype)
    assert ops.scaled_update(put32(x.clone()), put(o), None)[1] is None
    close(ops.rms_rows(put32(x), i32([4, 1], dev), w.to(dev), eps, dtype, groups), norm(x[[4, 1]]), dtype)
    if dev == "cuda":
        ops.nat().check_status()


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("T,E,k,d,ff", [(1, 4, 1, 32, 16), (5, 10, 3, 48, 24), (7, 6, 6, 45, 19), (64, 16, 4, 128, 136), (65, 12, 2, 256, 64), (700, 9, 2, 64, 48), (1500, 8, 4, 256, 256)])
def test_experts_whose_weight_multiplies_the_input(T, E, k, d, ff, dev, dtype):
    """Expert sort, gelu, sum without weights; a weight on the output instead would show."""
    x, up, down = rnd(T, d, seed=1), rnd(E, ff, d, seed=2, scale=0.8 * d ** -0.5), rnd(E, d, ff, seed=3, scale=3 * ff ** -0.5)
    g = torch.Generator().manual_seed(4)
    ids = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(T)]).int()
    wts = torch.rand(T, k, generator=g)
    want, other = torch.zeros(T, d, dtype=torch.float64), torch.zeros(T, d, dtype=torch.float64)
    for e in range(E):
        w = {"e.up": up[e].double(), "e.down": down[e].double()}
        for j in range(k):
            t = torch.nonzero(ids[:, j] == e).flatten()
            want[t] += O.expert(wts[t, j].double()[:, None] * x[t].double(), w, "e.")
            other[t] += wts[t, j].double()[:, None] * O.expert(x[t].double(), w, "e.")
    put = lambda t: t.to(dev, dtype)                                 # noqa: E731
    y, dest = ops.moe_routed(put(x), ids.to(dev), wts.to(dev), None, put(up), put(down))
    s, _, _ = ops.scaled_update(torch.zeros(T, d, device=dev), None, None, moe=(y, dest, None))
    close(s, want, dtype)
    assert (other - want).abs().max() > 0.01 * want.abs().max()


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("T,N,K", [(1, 40, 32), (9, 300, 72), (130, 520, 64), (3000, 1024, 256), (4, 7, 13)])
def test_exact_gelu_of_a_product(T, N, K, dev, dtype):
    x, w = rnd(T, K, seed=1), rnd(N, K, seed=2, scale=2.5 * K ** -0.5)
    y = ops.linear(x.to(dev, dtype), w.to(dev, dtype), unary=("gelu",))
    close(y, O.gelu(x.double() @ w.double().T), dtype)


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_sigmoid_router_keeps_its_scores(dev, dtype):
    T, E, top, d = 40, 12, 3, 64
    x, w = rnd(T, d, seed=1), rnd(E, d, seed=2, scale=2 * d ** -0.5)
    ids, wts = ops.moe_gate(x.to(dev, dtype), w.to(dev, dtype), None, top, 1, 1, 1.0, False, True, 2)
    got = torch.zeros(T, E + 2, dtype=torch.float64).scatter_(1, ids.long().cpu(), wts.double().cpu())
    close(got[:, :E], O.route(x.double() @ w.double().T, top), F32, scale=10)
    assert bool((got[:, E:] == 1).all()) and math.isclose(float(O.gelu(torch.tensor(1.0, dtype=torch.float64))), 0.8413447460685429)


def test_gathered_rows_count_whole_tiles_of_pooled_rows():
    from jittorinfer_b200.ops import native
    meta = {"total_kv": 5000, "q_lens": [500, 1, 30], "s_lens": [2000, 3000, 90]}
    seen = [len(O.seen_blocks(s - 1, 100, 16)) for s in meta["s_lens"]]
    assert seen == [118, 181, 0]
    assert native.visible_total(meta, 100, 0, 16) == 128 + 599 + 256 + 100 + 0 + 90 and native.visible_total(meta, 100) == 599 + 100 + 90
