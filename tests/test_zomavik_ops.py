"""Each mechanism of the Zomavik layers alone, against the plain oracle: the product's ops on the CPU and its kernels on a GPU."""
import pytest
import torch

import zomavik_oracle as O
from jittorinfer_b200 import ops
from jittorinfer_b200.models import folder
from jittorinfer_b200.ops.specs import Gqa, RowNorms, SelectiveScan

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


# ---- selective scan ------------------------------------------------------------------------------------------------------------
def run_scan(dev, dtype, ch, N, cuts, lens, slow=0.0, seed=0, single_ok=True):
    """Sequences interleaved in portions, alone and together, against the oracle on whole ones; slots hold what earlier sequences left."""
    neg_a, skip, bias = -torch.exp(rnd(ch, N, seed=seed + 1, scale=0.7)), rnd(ch, seed=seed + 2), rnd(ch, seed=seed + 3) - 2.0 - slow
    data = [[rnd(n, c, seed=50 + seed + 9 * j + i) for i, c in enumerate((ch, ch, 2 * N, ch))] for j, n in enumerate(lens)]      # x, z, B | C, dt
    want = []
    for x, z, bc, dt in ([t.double() for t in d] for d in data):
        y, S = O.selective_scan(x, O.softplus(dt + bias.double()), neg_a.double(), bc[:, :N], bc[:, N:], skip.double())
        want.append((y * O.silu(z) * 0.7, S))
    m = SelectiveScan(ch, N, neg_a.to(dev), skip.to(dev), bias.to(dev), 0.7)
    state = torch.full((4, ch, N), 3.0, device=dev)
    at, slots = [0] * len(lens), (3, 1)
    for cut in cuts:
        part = [(j, at[j], n) for j, n in enumerate(cut) if n]
        rows = torch.cat([torch.cat([t[p:p + n] for t in data[j]], 1) for j, p, n in part]).to(dev, dtype)
        x, z, bc, dt = torch.split(rows, [ch, ch, 2 * N, ch], 1)
        out = torch.full((rows.shape[0], ch + 8), 9.0, dtype=dtype, device=dev)
        single = single_ok and all(n == 1 for *_, n in part)
        ops.selective_scan(m, x, z, bc, dt, state, i32([slots[j] for j, *_ in part], dev), i32([p + k for _, p, n in part for k in range(n)], dev),
                           starts([n for *_, n in part], dev), single, out[:, 8:])
        close(out[:, 8:], torch.cat([want[j][0][p:p + n] for j, p, n in part]), dtype, f"cut {cut} at {at}")
        assert bool((out[:, :8] == 9).all())
        for j, _, n in part:
            at[j] += n
    assert tuple(at) == tuple(lens)
    for j in range(len(lens)):
        close(state[slots[j]], want[j][1], F32 if dtype == F32 else BF16, "state")
    assert bool((state[0] == 3).all()) and bool((state[2] == 3).all())
    if dev == "cuda":
        ops.nat().check_status()


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("ch,N", [(8, 8), (40, 16), (72, 24), (136, 32), (264, 64), (24, 128), (16, 200)])
def test_scan_in_portions_equals_one_pass(ch, N, dev, dtype):
    run_scan(dev, dtype, ch, N, [(1, 3), (1, 1), (2, 0), (67, 4), (1, 1), (0, 1), (16, 50), (17, 1), (1, 0), (44, 0)], (150, 61))
    run_scan(dev, dtype, ch, N, [(150, 0), (0, 61)], (150, 61), seed=1)
    run_scan(dev, dtype, ch, N, [(1, 1)] * 3 + [(5, 5)], (8, 8), seed=2, single_ok=False)


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_scan_remembers_over_long_prompts_and_long_decoding(dev, dtype):
    """Slow decays: what the first tokens wrote is still there; a lost or doubled update would stay."""
    run_scan(dev, dtype, 48, 16, [(260, 0), (0, 1)] + [(1, 1)] * 60, (320, 61), slow=4.0)
    run_scan(dev, dtype, 48, 32, [(129, 300), (191, 20)], (320, 320), slow=4.0)


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_scan_survives_very_fast_decays(dev, dtype):
    run_scan(dev, dtype, 48, 16, [(140, 61), (10, 0)], (150, 61), slow=-40.0)


@GPU
def test_scan_keeps_a_mark_among_a_thousand_tokens():
    """fp32: a state that hardly fades, one input that stands out a thousand tokens back, in one portion and token by token."""
    ch, N, n = 16, 16, 1100
    m = SelectiveScan(ch, N, torch.full((ch, N), -1e-3, device="cuda"), torch.zeros(ch, device="cuda"), torch.zeros(ch, device="cuda"))
    x, bc, dt = rnd(n, ch, seed=1, scale=1e-3), rnd(n, 2 * N, seed=2), torch.full((n, ch), -1.0)
    x[3] = 50.0
    z = torch.ones(n, ch)
    y, _ = O.selective_scan(x.double(), O.softplus(dt.double()), m.neg_a.double().cpu(), bc[:, :N].double(), bc[:, N:].double(), torch.zeros(ch).double())
    y = y * O.silu(z.double())
    for cuts in ([n], [700] + [1] * 400):
        st, got, p = torch.empty(1, ch, N, device="cuda"), [], 0
        for c in cuts:
            out = torch.empty(c, ch, device="cuda")
            f = lambda t: t[p:p + c].cuda()                          # noqa: B023,E731
            ops.selective_scan(m, f(x), f(z), f(bc), f(dt), st, i32([0], "cuda"), torch.arange(p, p + c, dtype=torch.int32, device="cuda"), i32([0, c], "cuda"), c == 1, out)
            got.append(out)
            p += c
        err = (torch.cat(got).cpu().double() - y).abs().max() / y.abs().max()
        assert err < 3e-6, err


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("single", [True, False])
def test_padding_rows_leave_states_alone(single, dev, dtype):
    ch, N = 24, 16
    st, cs = torch.full((2, ch, N), 5.0, device=dev), torch.full((2, 3, ch), 5.0, dtype=dtype, device=dev)
    m = SelectiveScan(ch, N, -torch.ones(ch, N, device=dev), torch.ones(ch, device=dev), torch.ones(ch, device=dev))
    x, bc, out = rnd(2, ch).to(dev, dtype), rnd(2, 2 * N).to(dev, dtype), torch.empty(2, ch, dtype=dtype, device=dev)
    args = (i32([-1, -1], dev), i32([0, 9], dev), i32([0, 1, 2], dev))
    ops.selective_scan(m, x, x, bc, x, st, *args, single, out)
    ops.causal_conv(x, rnd(4, ch).to(dev), cs, *args, rnd(ch).to(dev))
    assert bool((st == 5).all()) and bool((cs == 5).all())


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
def test_short_convolution_with_bias_and_silu(taps, dev, dtype):
    """A slice of the projection's columns; two sequences in portions; slots hold garbage."""
    ch, lens = 40, (50, 23)
    w, b = rnd(taps, ch, seed=1, scale=0.6), rnd(ch, seed=2, scale=0.3)
    seqs = [rnd(n, ch, seed=5 + j) for j, n in enumerate(lens)]
    want = [O.short_conv(s.double(), w.t().double(), b.double()) for s in seqs]
    state, at = torch.full((3, taps - 1, ch), 7.0, dtype=dtype, device=dev), [0, 0]
    for cut in ((1, 2), (2, 1), (1, 1), (17, 0), (1, 3), (3, 9), (25, 7)):
        part = [(j, at[j], n) for j, n in enumerate(cut) if n]
        x = torch.cat([seqs[j][p:p + n] for j, p, n in part])
        proj = torch.cat([rnd(x.shape[0], 16), x, rnd(x.shape[0], 8)], 1).to(dev, dtype)
        y = ops.causal_conv(proj[:, 16:16 + ch], w.to(dev), state, i32([2 * j for j, *_ in part], dev), i32([p + k for _, p, n in part for k in range(n)], dev),
                            starts([n for *_, n in part], dev), b.to(dev))
        close(y, torch.cat([want[j][p:p + n] for j, p, n in part]), dtype, f"{cut} at {at}")
        for j, _, n in part:
            at[j] += n
    assert tuple(at) == lens


# ---- attention -----------------------------------------------------------------------------------------------------------------
def run_attention(m, dev, dtype, cuts, lens, rot, seed=0, hot=(), want_prefill=None):
    """q, k, v through gqa_qkv_post and gqa_attention in portions over shuffled blocks, against the oracle on whole sequences.  ``hot``:
    (sequence, key) pairs whose keys every query likes."""
    H, G, D, V, bs = m.heads, m.kv_heads, m.dim, m.vdim, 64
    seqs = [[rnd(n, c, seed=30 + seed + 5 * j + i) for i, c in enumerate((H * D, G * D, G * V))] for j, n in enumerate(lens)]
    for j, p in hot:                                                 # along the unrotated last dimension
        seqs[j][0].view(lens[j], H, D)[..., -1] = 4.0 * D ** 0.5
        seqs[j][1].view(lens[j], G, D)[p] = 0
        seqs[j][1].view(lens[j], G, D)[p, :, -1] = 9.0
        seqs[j][2][p] = 3.0
    want = []
    for q, k, v in seqs:
        n = q.shape[0]
        qr, kr = O.rotate(q.double().view(n, H, D), rot), O.rotate(k.double().view(n, G, D), rot)
        sink = m.sink_w.double().cpu() if m.sink else torch.full((H,), -1e9, dtype=torch.float64)
        want.append((O.attend(qr, kr, v.double().view(n, G, V), m.scale, m.softcap, sink) * m.out_scale).reshape(n, H * V))
    nb = [(n + bs - 1) // bs for n in lens]
    perm = torch.randperm(sum(nb) + 2, generator=torch.Generator().manual_seed(3)).tolist()
    cache = torch.full(((sum(nb) + 2) * bs, m.kv_row), float("nan"), dtype=dtype, device=dev)
    tables = torch.zeros(len(lens), max(nb), dtype=torch.int32)
    for j, n in enumerate(nb):
        for i in range(n):
            tables[j, i] = perm.pop()
    md = Gqa(**{k: v.to(dev) if isinstance(v, torch.Tensor) else v for k, v in vars(m).items()})
    table = folder.rope_table(max(lens), folder.Rotation(rot["dims"], rot["base"]), dev)
    at, got = [0] * len(lens), [[] for _ in lens]
    before = ops.nat().launches_by_name.get("gqa_prefill", 0) if dev == "cuda" else 0
    for cut in cuts:
        part = [(j, at[j], n) for j, n in enumerate(cut) if n]
        proj = torch.cat([torch.cat([x[p:p + n] for x in seqs[j]], 1) for j, p, n in part]).to(dev, dtype)
        q_lens, s_lens = [n for *_, n in part], [p + n for _, p, n in part]
        slots = i32([int(tables[j, x // bs]) * bs + x % bs for j, p, n in part for x in range(p, p + n)], dev)
        a, b = H * D, (H + G) * D
        q = ops.gqa_qkv_post(md, proj[:, :a], proj[:, a:b], proj[:, b:], table, i32([p + k for _, p, n in part for k in range(n)], dev), slots, cache)
        out = torch.full((proj.shape[0], H * V + 8), 9.0, dtype=dtype, device=dev)
        meta = {"q_lens": q_lens, "s_lens": s_lens, "n_q_tiles": sum((x + 127) // 128 for x in q_lens), "total_kv": sum(s_lens), "kv_decode": 0}
        ops.gqa_attention(md, q, cache, None, tables[[j for j, *_ in part]].to(dev), i32(s_lens, dev), starts(q_lens, dev), bs, max(q_lens), meta, out[:, :H * V])
        assert bool((out[:, H * V:] == 9).all())
        k = 0
        for j, _, n in part:
            got[j].append(out[k:k + n, :H * V])
            at[j] += n
            k += n
    assert tuple(at) == tuple(lens)
    for j in range(len(lens)):
        close(torch.cat(got[j]), want[j], dtype, f"sequence {j}")
    if dev == "cuda":
        if want_prefill is not None:                                 # the tensor-core kernel ran where it should
            assert (ops.nat().launches_by_name.get("gqa_prefill", 0) > before) == (want_prefill and dtype == BF16)
        ops.nat().check_status()
    return want


def gqa(H=4, G=2, D=24, V=20, rot=16, softcap=11.0, scale=None, sink=1.5, **kw):
    return Gqa(H, G, D, V, rot, D ** -0.5 if scale is None else scale, softcap=softcap, sink=True, sink_w=rnd(H, seed=77, scale=sink), out_scale=0.7, **kw)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("shape", [dict(), dict(H=1, G=1, D=8, V=8, rot=2), dict(H=21, G=1, D=13, V=9, rot=6), dict(H=8, G=8, D=64, V=64, rot=64, softcap=0.0),
                                   dict(H=3, G=3, D=40, V=200, rot=20), dict(H=34, G=2, D=96, V=36, rot=48), dict(H=6, G=1, D=48, V=96, rot=32),
                                   dict(H=4, G=2, D=128, V=128, rot=128), dict(H=6, G=2, D=128, V=128, rot=64, softcap=0.0)])
def test_attention_in_portions_equals_one_pass(shape, dev, dtype):
    m = gqa(**shape)
    rot = dict(dims=m.rot, base=900.0)
    wide = m.dim == m.vdim == 128
    run_attention(m, dev, dtype, [(1, 2), (1, 1), (130, 3), (1, 1), (2, 60), (65, 33), (40, 0)], (240, 100), rot, want_prefill=wide)
    run_attention(gqa(**shape), dev, dtype, [(240, 0), (0, 100)], (240, 100), rot, seed=1, want_prefill=wide)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("D", [24, 32, 128])
def test_far_keys_among_many(D, dev, dtype):
    """One key among a thousand far behind the queries, at block borders too."""
    run_attention(gqa(D=D, V=D, softcap=25.0), dev, dtype, [(1, 0), (1000, 0), (1, 0), (3, 0), (1, 0), (0, 1)], (1006, 1), dict(dims=16, base=900.0),
                  hot=[(0, 5), (0, 63), (0, 64)])


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("D", [24, 32, 128])
def test_sinks_of_any_size_count_once(D, dev, dtype):
    """Sinks far above and far below every score, in prompts, split decoding and the first tokens; the softmax neither overflows nor
    forgets them, and another sink shows."""
    for value in (-60.0, 0.0, 9.0, 60.0):
        m = gqa(D=D, V=D)
        m.sink_w = torch.tensor([value, -value, value / 3, 0.0])
        want = run_attention(m, dev, dtype, [(300, 1), (1, 1), (2, 1), (1, 67)], (304, 70), dict(dims=16, base=900.0))
        first = want[0][0].view(4, D).abs().amax(-1)                 # position 0: one key beside the sink
        assert value < 50 or (first[0] < 1e-9 and first[1] > 0.1)


# ---- routing -------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("T", [1, 5, 70, 600])
@pytest.mark.parametrize("d,E,top,groups,shared", [(48, 12, 3, (3, 2), 1), (64, 16, 4, (2, 1), 2), (43, 15, 5, (5, 3), 0), (1032, 64, 6, None, 2), (32, 1, 1, None, 1), (256, 160, 6, (8, 3), 0)])
def test_router_with_groups_and_a_gated_shared_expert(d, E, top, groups, shared, T, dev, dtype):
    h, w = rnd(T, d, seed=1), rnd(E + 1, d, seed=2, scale=2 * d ** -0.5)
    z = h.double() @ w.double().T
    want = O.route(z[:, :E], top, dict(count=groups[0], keep=groups[1]) if groups else None)
    for wd in (w.to(dev), w.to(dev, dtype)):
        c, k = groups or (1, 1)
        ids, wts, gate = ops.moe_gate(h.to(dev, dtype), wd, None, top, c, k, 1.0, True, False, shared, shared_gate=True)
        got = torch.zeros(T, E + 1).scatter_add_(1, ids[:, :top].long().cpu(), wts[:, :top].cpu())
        close(got[:, :E], want, F32)
        close(gate, z[:, E], F32)
        if shared:
            assert ids[:, top:].tolist() == [list(range(E, E + shared))] * T
            close(wts[:, top:], torch.sigmoid(z[:, E:]).expand(T, shared), F32)


# ---- rows and products -------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("d", [24, 43, 1032, 2056, 5128, 8200])
def test_scaled_updates_with_one_norm_two_or_none(d, dev, dtype):
    T, k = 5, 3
    table, ids = rnd(11, d, seed=1), [3, 0, 10, 7, 7]
    w1, w2, s1, s2 = (rnd(d, seed=2 + i, scale=0.2, mean=1.0).to(dev) for i in range(4))
    two, one, none = RowNorms(1e-3, w1, w2), RowNorms(1e-3, w1), RowNorms()
    x, h, h2 = ops.embed_norm(table.to(dev, dtype), i32(ids, dev), None, 1e-3, two, 1.7)
    want = table[ids] * 1.7
    close(x, want, F32)
    close(h, O.norm(want, w1.cpu(), 1e-3), dtype)
    close(h2, O.norm(want, w2.cpu(), 1e-3), dtype)
    _, h, h2 = ops.embed_norm(table.to(dev, dtype), i32(ids, dev), None, 1e-3, none, 1.7)
    close(h, want, dtype)
    assert h2 is None and h.dtype == dtype
    o, y, f = (rnd(n, d, seed=10 + n).to(dev, dtype) for n in (T, T * k, T + 1))
    f, gate = f[:T].contiguous(), rnd(T, 3, seed=20).to(dev)[:, 1]
    dest = torch.randperm(T * k, generator=torch.Generator().manual_seed(0)).int().view(T, k).to(dev)
    wts = rnd(T, k, seed=21).abs().to(dev)
    ro, ry, rf = (t.float().cpu() for t in (o, y, f))
    routed = (ry[dest.cpu().long()] * wts.cpu()[..., None]).sum(1)
    gated = torch.sigmoid(gate.cpu())[:, None] * rf
    for moe, dense, dg, sub in ((None, None, None, None), (None, f, None, rf), ((y, dest, wts), None, None, routed), ((y, dest, wts), f, gate, routed + gated)):
        for nxt in (two, one, none, None):
            xo, h, h2 = ops.scaled_update(x.clone(), o, s1, s2, moe=moe, dense=dense, dense_gate=dg, nxt=nxt)
            v = want + s1.cpu() * ro + (s2.cpu() * sub if sub is not None else 0)
            close(xo, v, F32)
            assert (h is None) == (nxt is None) and (h2 is None) == (nxt is not two)
            if nxt is not None:
                close(h, v if nxt is none else O.norm(v, w1.cpu(), 1e-3), dtype)
            if nxt is two:
                close(h2, O.norm(v, w2.cpu(), 1e-3), dtype)
    xo, h, h2 = ops.scaled_update(x.clone(), None, None, nxt=two, dtype=dtype)       # norms alone
    close(xo, want, F32)
    close(h2, O.norm(want, w2.cpu(), 1e-3), dtype)


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("T,d,n", [(1, 64, 72), (5, 43, 29), (70, 256, 520), (300, 128, 384), (700, 512, 1024), (600, 1032, 160), (520, 2048, 65)])
def test_functions_and_biases_of_single_products(T, d, n, dev, dtype):
    x, w, b = rnd(T, d, seed=1), rnd(n, d, seed=2, scale=2 * d ** -0.5), rnd(n, seed=3)
    y = x.double() @ w.double().T
    args = [t.to(dev, dtype) for t in (x, w)]
    close(ops.linear(*args, unary=("relu2",)), torch.relu(y) ** 2, dtype)
    for scale, cap in ((0.5, 3.0), (2.0, 0.7), (0.3, 0.0), (40.0, 5.0)):
        for od in (F32, dtype):
            close(ops.linear(*args, out_dtype=od, unary=("cap", scale, cap)), O.capped(y * scale, cap), od)
    close(ops.linear(*args, residual=b.to(dev).expand(T, -1)), y + b, dtype)
    close(ops.linear(*args, residual=rnd(T, n, seed=4).to(dev), out_dtype=F32), y + rnd(T, n, seed=4), F32 if dtype == F32 else BF16)
