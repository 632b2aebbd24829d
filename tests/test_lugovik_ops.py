"""Each mechanism of the Lugovik layers alone, against the plain oracle: the product's ops on the CPU and its kernels on a GPU."""
import math

import pytest
import torch

import lugovik_oracle as O
from jittorinfer_b200 import ops
from jittorinfer_b200.models import lugovik
from jittorinfer_b200.ops.specs import Gqa, StateMix

GPU = pytest.mark.gpu
WHERE = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda", torch.float32, id="cuda-f32", marks=GPU),
         pytest.param("cuda", torch.bfloat16, id="cuda-bf16", marks=GPU)]
F32, BF16 = torch.float32, torch.bfloat16


def tol(dtype):
    return 3e-5 if dtype == F32 else 2.5e-2


def close(a, b, dtype, what=""):
    a, b = a.double().cpu(), b.double().cpu()
    err = (a - b).abs().max().item()
    assert err <= tol(dtype) * max(1.0, b.abs().max().item()), f"{what}: {err} of {b.abs().max().item()}"


def rnd(*shape, seed=0, scale=1.0, mean=0.0):
    return (mean + torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * scale).bfloat16().float()


def i32(x, dev="cpu"):
    return torch.tensor(x, dtype=torch.int32, device=dev)


# ---- matrix-state mixers -------------------------------------------------------------------------------------------------------
def state_case(kind, H, K, V, rep, taps, groups=1, slow=0.0, seed=0):
    """(StateMix on the CPU, columns of proj, function (proj, dec_in, gate) -> (y, final state) by the oracle)."""
    Hk = H // rep
    off, cols = {}, 0
    order = (("v", H * V), ("k", Hk * K), ("q", Hk * K), ("s", H)) if kind == "ssd" else (("q", Hk * K), ("k", Hk * K), ("v", H * V), ("s", H))
    for name, n in order:
        off[name] = cols
        cols += n
    n_conv = off["s"]
    cols = (cols + 7) // 8 * 8
    per_head = kind == "ssd"
    m = StateMix(kind, H, K, V, rep, q_off=off["q"], k_off=off["k"], v_off=off["v"], s_off=off["s"], taps=taps, norm_groups=groups,
                 q_scale=1.0 if kind == "ssd" else K ** -0.5, inv_tau=1 / 7.0, eps=1e-2, out_scale=1.3)
    if taps:
        m.conv_w = rnd(taps, n_conv, seed=seed + 1, scale=0.7)
        m.conv_b = rnd(n_conv, seed=seed + 2, scale=0.3) if kind == "ssd" else None
    m.bias = rnd(H if per_head else H * K, seed=seed + 3) + (slow if kind == "linear" else -2.0 - slow)
    m.neg_a = -torch.exp(rnd(H, seed=seed + 4, scale=0.7))
    m.skip = rnd(H, seed=seed + 5)
    m.norm_w = rnd(H * V if per_head else V, seed=seed + 6, scale=0.2, mean=1.0)

    def oracle(proj, dec_in, gate):
        proj, dec_in, gate = proj.double(), dec_in.double(), gate.double()
        n = proj.shape[0]
        x = O.short_conv(proj[:, :n_conv], m.conv_w.t().double(), None if m.conv_b is None else m.conv_b.double()) if taps else proj
        head = torch.arange(H) // rep
        q, k = (x[:, off[c]:off[c] + Hk * K].view(n, Hk, K)[:, head] for c in "qk")
        v = x[:, off["v"]:off["v"] + H * V].view(n, H, V)
        s = proj[:, off["s"]:off["s"] + H]
        if kind == "ssd":
            dt = O.softplus(s + m.bias)
            o, S = O.linear_state(q, k, dt[..., None] * v, torch.exp(m.neg_a.double() * dt)[..., None].expand(n, H, K))
            y = ((o + m.skip.double()[:, None] * v).reshape(n, H * V) * O.silu(gate)).view(n, groups, -1)
            return O.norm(y, m.norm_w.double().view(groups, -1), m.eps).reshape(n, H * V) * m.out_scale, S
        z = (dec_in + m.bias).view(n, H, K)
        if kind == "delta":
            dec = torch.exp(m.neg_a.double()[:, None] * O.softplus(z))
            o, S = O.delta_state(O.unit(q) * m.q_scale, O.unit(k), v, dec, torch.sigmoid(s))
            return (O.norm(o, m.norm_w.double(), m.eps).reshape(n, H * V) * torch.sigmoid(gate)) * m.out_scale, S
        o, S = O.linear_state(q * m.q_scale, k, v, torch.sigmoid(z) ** m.inv_tau)
        return O.norm(o, m.norm_w.double(), m.eps).reshape(n, H * V) * O.silu(gate) * m.out_scale, S
    return m, cols, n_conv, oracle


def to_dev(m, dev):
    return StateMix(**{k: v.to(dev) if isinstance(v, torch.Tensor) else v for k, v in vars(m).items()})


SIZES = {"small": dict(H=4, K=20, V=28, rep=2, taps=4), "odd": dict(H=6, K=11, V=7, rep=3, taps=6), "one": dict(H=1, K=1, V=1, rep=1, taps=1),
         "head": dict(H=2, K=128, V=128, rep=1, taps=4), "wide": dict(H=2, K=80, V=160, rep=2, taps=2), "deep": dict(H=1, K=300, V=36, rep=1, taps=3),
         "groups": dict(H=6, K=64, V=40, rep=2, taps=3), "large": dict(H=1, K=256, V=256, rep=1, taps=0), "tile": dict(H=4, K=64, V=48, rep=2, taps=3),
         "bare": dict(H=2, K=128, V=16, rep=1, taps=0), "block": dict(H=2, K=64, V=256, rep=1, taps=1)}
TENSOR_CORE = ("head", "tile", "bare", "block")                     # sizes the chunked kernels are built for


def run_state(kind, dev, dtype, size, cuts, slow=0.0, lens=(150, 61), single_ok=True, seed=0):
    z = SIZES[size]
    m, cols, n_conv, oracle = state_case(kind, **z, groups=2 if kind == "ssd" and z["H"] % 2 == 0 else 1, slow=slow, seed=seed)
    H, K, V = m.heads, m.dim, m.vdim
    data = [[rnd(n, c, seed=50 + seed + 7 * j + i) for i, c in enumerate((cols, H * K, H * V))] for j, n in enumerate(lens)]
    want = [oracle(*d) for d in data]
    md = to_dev(m, dev)
    state = torch.full((4, H, K, V), 3.0, device=dev)                # whatever earlier sequences left
    conv = torch.full((4, max(m.taps, 1), n_conv), 5.0, dtype=dtype, device=dev) if m.taps else None
    at = [0] * len(lens)
    slots = (3, 1)
    chunked = ops.nat().launches_by_name.get("state_chunk", 0) if dev == "cuda" else 0
    for cut in cuts:
        part = [(j, at[j], n) for j, n in enumerate(cut) if n]
        proj, dec, gate = (torch.cat([data[j][c][p:p + n] for j, p, n in part]).to(dev, dtype) for c in range(3))
        pos = i32([p + k for _, p, n in part for k in range(n)], dev)
        qs = i32([0] + torch.tensor([n for *_, n in part]).cumsum(0).tolist(), dev)
        out = torch.full((proj.shape[0], H * V + 8), 9.0, dtype=dtype, device=dev)
        single = single_ok and all(n == 1 for *_, n in part)
        ops.state_mix(md, proj, None if kind == "ssd" else dec, gate, conv, state, i32([slots[j] for j, *_ in part], dev), pos, qs, single, out[:, 8:])
        close(out[:, 8:], torch.cat([want[j][0][p:p + n] for j, p, n in part]), dtype, f"cut {cut} at {at}")
        assert bool((out[:, :8] == 9).all())
        for j, _, n in part:
            at[j] += n
    assert tuple(at) == tuple(lens)
    for j in range(len(lens)):
        close(state[slots[j]], want[j][1], F32 if dtype == F32 else BF16, "state")
    assert bool((state[0] == 3).all()) and bool((state[2] == 3).all())
    if dev == "cuda":
        assert (ops.nat().launches_by_name.get("state_chunk", 0) > chunked) == (dtype == BF16 and size in TENSOR_CORE)
        ops.nat().check_status()
    if m.taps > 1:                                                   # the ring holds the last inputs, row p % taps
        for j in range(len(lens)):
            for d in range(1, m.taps):
                close(conv[slots[j], (lens[j] - d) % m.taps], data[j][0][lens[j] - d, :n_conv], dtype, "ring")
        assert bool((conv[0] == 5).all())


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("size", list(SIZES))
@pytest.mark.parametrize("kind", ["delta", "linear", "ssd"])
def test_state_mix_in_portions_equals_one_pass(kind, size, dev, dtype):
    """Two sequences interleaved in portions down to one token, alone and together; the slots hold garbage from earlier sequences."""
    run_state(kind, dev, dtype, size, [(1, 3), (1, 1), (2, 0), (67, 4), (1, 1), (0, 1), (16, 50), (17, 1), (1, 0), (44, 0)])


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("kind", ["delta", "linear", "ssd"])
def test_state_mix_remembers_over_long_prompts_and_long_decoding(kind, dev, dtype):
    """Slow decays: what the first tokens wrote is still there; a lost or doubled update would stay."""
    for size in ("small", "head"):
        run_state(kind, dev, dtype, size, [(260, 0), (0, 1)] + [(1, 1)] * 60, slow=4.0, lens=(320, 61))
        run_state(kind, dev, dtype, size, [(129, 300), (191, 20)], slow=4.0, lens=(320, 320))


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("kind", ["delta", "linear", "ssd"])
def test_state_mix_survives_very_fast_decays(kind, dev, dtype):
    """Decays down to zero: products over a few tokens underflow, their quotients must not matter."""
    for size in ("small", "head"):
        run_state(kind, dev, dtype, size, [(140, 61), (10, 0)], slow=-8.0 if kind != "linear" else -90.0)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("kind", ["delta", "linear", "ssd"])
def test_padding_rows_leave_every_state_alone(kind, dev, dtype):
    m, cols, n_conv, _ = state_case(kind, **SIZES["small"])
    H, K, V = m.heads, m.dim, m.vdim
    st, cs = torch.full((2, H, K, V), 5.0, device=dev), torch.full((2, m.taps, n_conv), 5.0, dtype=dtype, device=dev)
    for single in (True, False):
        out = torch.empty(2, H * V, dtype=dtype, device=dev)
        ops.state_mix(to_dev(m, dev), rnd(2, cols).to(dev, dtype), rnd(2, H * K).to(dev, dtype), rnd(2, H * V).to(dev, dtype), cs, st,
                      i32([-1, -1], dev), i32([0, 9], dev), i32([0, 1, 2], dev), single, out)
    assert bool((st == 5).all()) and bool((cs == 5).all())


# ---- rotation --------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("scaling", [None, (4.0, 96, 8.0, 1.0), (8.0, 32, 30.0, 4.0), (1.0, 64, 32.0, 1.0), (2.5, 10 ** 6, 2.0, 1.5)])
@pytest.mark.parametrize("dims", [2, 12, 64])
def test_rotation_table_blends_frequencies(dims, scaling):
    yarn = None if scaling is None else lugovik.Yarn(*scaling)
    t = lugovik.rope_table(300, lugovik.Rotation(dims, 700.0, yarn), "cpu")
    f, mult = O.frequencies(dims, 700.0, None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling)))
    for p in (0, 1, 77, 299):
        for i in range(dims // 2):
            assert abs(t[p, i, 0] - mult * math.cos(p * f[i])) < 1e-6 and abs(t[p, i, 1] - mult * math.sin(p * f[i])) < 1e-6


# ---- attention -------------------------------------------------------------------------------------------------------------------
class Paged:
    """Two sequences over shuffled blocks of one cache whose other rows are NaN."""

    def __init__(self, m, lens, dtype, dev, bs=64):
        nb = [(n + bs - 1) // bs for n in lens]
        perm = torch.randperm(sum(nb) + 2, generator=torch.Generator().manual_seed(3)).tolist()
        self.cache = torch.full(((sum(nb) + 2) * bs, m.kv_row), float("nan"), dtype=dtype, device=dev)
        self.tables, self.bs, self.dev = torch.zeros(len(lens), max(nb), dtype=torch.int32), bs, dev
        for j, n in enumerate(nb):
            for i in range(n):
                self.tables[j, i] = perm.pop()

    def slots(self, j, pos):
        return [int(self.tables[j, p // self.bs]) * self.bs + p % self.bs for p in pos]


def run_attention(m, dev, dtype, cuts, lens, rot, seed=0, hot=()):
    """q, k, v through gqa_qkv_post and gqa_attention in portions, against the oracle on whole sequences.  ``hot``: (sequence, key) pairs whose
    keys every later query likes."""
    H, G, D, V = m.heads, m.kv_heads, m.dim, m.vdim
    m.q_norm, m.k_norm = rnd(D, seed=1, scale=0.2, mean=1.0), rnd(D, seed=2, scale=0.2, mean=1.0)
    seqs = [[rnd(n, c, seed=30 + seed + 5 * j + i) for i, c in enumerate((H * D, G * D, G * V, H))] for j, n in enumerate(lens)]
    for j, p in hot:                                                 # along the unrotated last dimension
        for q in seqs[j][0].view(lens[j], H, D):
            q[:, -1] = 4.0 * D ** 0.5
        seqs[j][1].view(lens[j], G, D)[p] = 0
        seqs[j][1].view(lens[j], G, D)[p, :, -1] = 9.0
        seqs[j][2][p] = 3.0
    want = []
    for q, k, v, g in seqs:
        n = q.shape[0]
        pos = torch.arange(n)
        qr = O.rotate(O.norm(q.double().view(n, H, D), m.q_norm.double(), m.eps), pos, rot)
        kr = O.rotate(O.norm(k.double().view(n, G, D), m.k_norm.double(), m.eps), pos, rot)
        o = O.attend(qr, kr, v.double().view(n, G, V), m.scale, m.softcap, m.chunk)
        want.append((o * torch.sigmoid(g.double())[..., None] * m.out_scale).reshape(n, H * V))
    pg = Paged(m, lens, dtype, dev)
    md = Gqa(**{k: v.to(dev) if isinstance(v, torch.Tensor) else v for k, v in vars(m).items()})
    sc = rot.get("scaling")
    table = lugovik.rope_table(max(lens), lugovik.Rotation(rot["dims"], rot["base"], None if sc is None else lugovik.Yarn(**sc)), dev)
    at, got = [0] * len(lens), [[] for _ in lens]
    prefills = ops.nat().launches_by_name.get("gqa_prefill", 0) if dev == "cuda" else 0
    for cut in cuts:
        part = [(j, at[j], n) for j, n in enumerate(cut) if n]
        proj = torch.cat([torch.cat([x[p:p + n] for x in seqs[j]], 1) for j, p, n in part]).to(dev, dtype)
        pos = i32([p + k for _, p, n in part for k in range(n)], dev)
        slots = i32([s for j, p, n in part for s in pg.slots(j, range(p, p + n))], dev)
        q_lens = [n for *_, n in part]
        s_lens = [p + n for _, p, n in part]
        qs = i32([0] + torch.tensor(q_lens).cumsum(0).tolist(), dev)
        a, b, c = H * D, (H + G) * D, (H + G) * D + G * V
        q = ops.gqa_qkv_post(md, proj[:, :a], proj[:, a:b], proj[:, b:c], table, pos, slots, pg.cache)
        out = torch.full((proj.shape[0], H * V + 8), 9.0, dtype=dtype, device=dev)
        meta = {"q_lens": q_lens, "s_lens": s_lens, "n_q_tiles": sum((x + 127) // 128 for x in q_lens), "total_kv": sum(s_lens), "kv_decode": 0}
        ops.gqa_attention(md, q, pg.cache, proj[:, c:], pg.tables[[j for j, *_ in part]].to(dev), i32(s_lens, dev), qs, 64, max(q_lens), meta, out[:, :H * V])
        assert bool((out[:, H * V:] == 9).all())
        k = 0
        for j, _, n in part:
            got[j].append(out[k:k + n, :H * V])
            at[j] += n
            k += n
    assert tuple(at) == tuple(lens)
    for j in range(len(lens)):
        close(torch.cat(got[j]), want[j], dtype, f"sequence {j}")
    if dev == "cuda":                                                # the tensor-core kernel ran where it should
        assert (ops.nat().launches_by_name.get("gqa_prefill", 0) > prefills) == (dtype == BF16 and D == V == 128 and max(map(sum, cuts)) >= 64)
        ops.nat().check_status()
    return want


def gqa(H=4, G=2, D=24, V=20, rot=16, chunk=50, softcap=11.0, scale=None, **kw):
    return Gqa(H, G, D, V, rot, D ** -0.5 if scale is None else scale, softcap=softcap, chunk=chunk, sink=True, eps=1e-4, out_scale=0.7, **kw)


YARN = dict(factor=3.0, original=96, fast=8.0, slow=1.0)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("shape", [dict(), dict(H=1, G=1, D=8, V=8, rot=2, chunk=3), dict(H=21, G=1, D=13, V=9, rot=6, chunk=37), dict(H=8, G=8, D=64, V=64, rot=64, chunk=64),
                                   dict(H=3, G=3, D=40, V=200, rot=20, chunk=1000), dict(H=34, G=2, D=96, V=36, rot=48, chunk=130), dict(H=2, G=1, D=260, V=300, rot=64, chunk=70),
                                   dict(H=4, G=2, D=128, V=128, rot=128, chunk=96), dict(H=6, G=2, D=128, V=128, rot=64, chunk=512)])
def test_attention_in_portions_equals_one_pass(shape, dev, dtype):
    m = gqa(**shape)
    rot = dict(dims=m.rot, base=900.0, **({"scaling": YARN} if m.heads % 2 == 0 else {}))
    run_attention(m, dev, dtype, [(1, 2), (1, 1), (130, 3), (1, 1), (2, 60), (65, 33), (40, 0)], (240, 100), rot)
    run_attention(gqa(**shape), dev, dtype, [(240, 0), (0, 100)], (240, 100), rot, seed=1)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("D", [24, 128])
@pytest.mark.parametrize("chunk", [63, 64, 65, 128, 40, 129])
def test_the_chunks_edge_shows(chunk, D, dev, dtype):
    """The last key of a chunk and the first of the next stand out: later queries of their chunk see little else, others nothing of
    them.  In prompts, in portions that end at the edge, and in decoding across it."""
    n = 2 * chunk + 10
    hot = [(0, chunk - 1), (0, chunk), (1, 0), (1, chunk + 3), (1, 2 * chunk - 1)]
    rot = dict(dims=16, base=900.0)
    for cuts in ([(n, n)], [(chunk - 2, chunk + 1)] + [(1, 1)] * 5 + [(chunk + 7, chunk + 4)], [(chunk, 2 * chunk)] + [(1, 1)] * 9 + [(chunk + 1, 1)]):
        want = run_attention(gqa(chunk=chunk, D=D, V=D, softcap=20.0), dev, dtype, cuts, (n, n), rot, hot=hot)
    assert want[0][chunk - 1].abs().max() > 0.5 and want[0][chunk + 1].abs().max() > 0.5       # they do stand out


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_far_keys_among_many(dev, dtype):
    """One key among a thousand, in one chunk, far behind the queries."""
    for D in (24, 128):
        run_attention(gqa(chunk=2000, D=D, V=D, softcap=25.0), dev, dtype, [(1, 0), (1000, 0), (1, 0), (3, 0), (1, 0), (0, 1)], (1006, 1), dict(dims=16, base=900.0), hot=[(0, 5)])


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("window,chunk,cap,sink,gated", [(0, 0, 0.0, False, False), (70, 0, 0.0, True, True), (30, 50, 8.0, False, True)])
def test_attention_options_of_other_designs(window, chunk, cap, sink, gated, dev, dtype):
    """No chunks, a sliding window, both, no cap, no sink, no gate."""
    H, G, D, V, n = 4, 2, 24, 20, 150
    m = Gqa(H, G, D, V, 0, 0.3, softcap=cap, window=window, chunk=chunk, sink=sink, eps=1e-4)
    q, k, v, g = rnd(n, H, D, seed=1), rnd(n, G, D, seed=2), rnd(n, G, V, seed=3), rnd(n, H, seed=4)
    want = torch.zeros(n, H, V, dtype=torch.float64)
    for i in range(n):
        js = [j for j in range(i + 1) if (not window or i - j < window) and (not chunk or i // chunk == j // chunk)]
        for h in range(H):
            s = (k[js, h // 2].double() @ q[i, h].double()) * m.scale
            s = cap * torch.tanh(s / cap) if cap else s
            e = torch.exp(s)
            want[i, h] = (e @ v[js, h // 2].double()) / (e.sum() + (1 if sink else 0))
            if gated:
                want[i, h] *= torch.sigmoid(g[i, h].double())
    pg = Paged(m, (n,), dtype, dev)
    pg.cache[pg.slots(0, range(n))] = torch.cat([k.reshape(n, -1), v.reshape(n, -1)], 1).to(dev, dtype)
    for lo, hi in ((0, n), (100, n), (n - 1, n)):
        out = torch.zeros(hi - lo, H * V, dtype=dtype, device=dev)
        ops.gqa_attention(m, q[lo:hi].to(dev, dtype).contiguous(), pg.cache, g[lo:hi].to(dev, dtype) if gated else None, pg.tables.to(dev), i32([hi], dev),
                          i32([0, hi - lo], dev), 64, hi - lo, None, out)
        close(out, want[lo:hi].reshape(hi - lo, H * V), dtype)


# ---- rows: embedding, norms around a sublayer, gated feed-forward ------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("d", [24, 43, 1032, 2056, 5128, 8200])
def test_scaled_embedding_and_norms_around_a_sublayer(d, dev, dtype):
    T = 5
    table, ids = rnd(11, d, seed=1), [3, 0, 10, 7, 7]
    w1, w2 = rnd(d, seed=2, scale=0.2, mean=1.0), rnd(d, seed=3, scale=0.2, mean=1.0)
    x, h, hc = ops.embed_norm(table.to(dev, dtype), i32(ids, dev), None, 1e-3, (w1.to(dev), 1e-3, None), 3.7)
    want = table[ids] * 3.7
    close(x, want, F32, "the residual stays fp32")
    close(h, O.norm(want, w1, 1e-3), dtype)
    assert x.dtype == F32 and hc is None
    y = rnd(T, d, seed=4, scale=5.0)
    want = want + O.norm(y, w2, 1e-3)
    xo, h = ops.post_norm(x.clone(), y.to(dev, dtype), w2.to(dev), 1e-3, (w1.to(dev), 1e-2, None))
    close(xo, want, F32)
    close(h, O.norm(want, w1, 1e-2), dtype)
    xo, h = ops.post_norm(x.clone(), y.to(dev, dtype), w2.to(dev), 1e-3)
    close(xo, want, F32)
    assert h is None
    close(ops.rms_rows(xo, i32([4, 1], dev), w1.to(dev), 1e-3, dtype), O.norm(want[[4, 1]], w1, 1e-3), dtype)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("T,d,ff", [(1, 64, 72), (5, 43, 29), (70, 256, 520), (300, 128, 384), (700, 512, 1024)])
def test_gelu_gate(T, d, ff, dev, dtype):
    x, g, u = rnd(T, d, seed=1), rnd(ff, d, seed=2, scale=2 * d ** -0.5), rnd(ff, d, seed=3, scale=d ** -0.5)
    want = O.gelu_tanh(x @ g.T) * (x @ u.T)
    args = [t.to(dev, dtype) for t in (x, g, u)]
    close(ops.gateup(*args, "gelu_tanh"), want, dtype)
    close(ops.gateup(*args, "silu"), O.silu(x @ g.T) * (x @ u.T), dtype)
