"""Each mechanism of the Nibalix layers alone, against the plain oracle: the product's ops on the CPU and its kernels on a GPU."""
import pytest
import torch

import nibalix_oracle as O
from jittorinfer_b200 import ops

GPU = pytest.mark.gpu
WHERE = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda", torch.float32, id="cuda-f32", marks=GPU),
         pytest.param("cuda", torch.bfloat16, id="cuda-bf16", marks=GPU)]
F32, BF16 = torch.float32, torch.bfloat16


def tol(dtype):
    return 3e-5 if dtype == F32 else 2.5e-2


def close(a, b, dtype, what=""):
    a, b = a.double().cpu(), b.double().cpu()
    err = (a - b).abs().max().item()
    assert err <= tol(dtype) * max(1.0, b.abs().max().item()), f"{what}: {err}"


def rnd(*shape, seed=0, scale=1.0):
    return (torch.randn(shape, generator=torch.Generator().manual_seed(seed)) * scale).bfloat16().float()


def i32(x, dev="cpu"):
    return torch.tensor(x, dtype=torch.int32, device=dev)


def ranges(cuts):
    """Portions of one sequence as (first position, length)."""
    out, p = [], 0
    for n in cuts:
        out.append((p, n))
        p += n
    return out


# ---- convolution ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_causal_conv_in_portions_with_reused_slots(dev, dtype, taps):
    """Two sequences interleaved in portions down to one token; the slots hold garbage from earlier sequences."""
    d = 24
    seqs = [rnd(29, d, seed=1), rnd(40, d, seed=2)]
    w = rnd(d, taps, seed=3)
    want = [h + O.input_conv(h, w) for h in seqs]
    state = torch.full((3, taps - 1, d), 7.0, dtype=dtype, device=dev)
    wt = w.t().contiguous().to(dev)
    at = [0, 0]
    for cut in [(2, 5), (1, 1), (0, 2), (3, 0), (9, 2), (14, 30)]:
        part = [(s, at[s], n) for s, n in enumerate(cut) if n]
        h = torch.cat([seqs[s][p:p + n] for s, p, n in part]).to(dev, dtype)
        pos = i32([p + k for _, p, n in part for k in range(n)], dev)
        qs = i32([0] + torch.tensor([n for *_, n in part]).cumsum(0).tolist(), dev)
        out = ops.causal_conv(h, wt, state, i32([(2, 0)[s] for s, *_ in part], dev), pos, qs)
        ref = torch.cat([want[s][p:p + n] for s, p, n in part])
        close(out, ref, dtype, f"cut {cut}")
        for s, _, n in part:
            at[s] += n
    assert at == [29, 40]
    if taps > 1:
        close(state[2], seqs[0][29 - taps + 1:], dtype, "stored rows")
        assert bool((state[1] == 7).all())                        # a slot nobody used


# ---- recurrence ----------------------------------------------------------------------------------------------------------------
def _gru_ref(zxg, zb, xb, s0=None):
    W = zb.shape[0]
    z, u, g = (zxg[:, k * W:(k + 1) * W].double() for k in range(3))
    z, u = torch.sigmoid(z + zb), u + xb
    c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    s = torch.zeros(W, dtype=torch.float64) if s0 is None else s0
    ys = []
    for t in range(zxg.shape[0]):
        s = (1 - z[t]) * s + z[t] * c[t]
        ys.append(s * g[t] * torch.sigmoid(g[t]))
    return torch.stack(ys), s


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("W", [16, 33, 200])
def test_mingru_in_portions_equals_one_pass(dev, dtype, W):
    """Portions around the scan's run, chunk and round lengths (4, 128, 1024), single tokens, two sequences, slots with old states; the state
    is slow to forget (gates near 0), so an error in the carry would stay."""
    lens = (1300, 61)
    zxg = [rnd(n, 3 * W, seed=10 + i) for i, n in enumerate(lens)]
    zb, xb = rnd(W, seed=4) - 5.0, rnd(W, seed=5)
    want = [_gru_ref(x, zb, xb) for x in zxg]
    state = torch.full((4, W), -3.0, device=dev)
    at = [0, 0]
    for cut in [(1, 3), (2, 0), (1027, 4), (1, 1), (129, 50), (128, 3), (12, 0)]:
        part = [(s, at[s], n) for s, n in enumerate(cut) if n]
        x = torch.cat([zxg[s][p:p + n] for s, p, n in part]).to(dev, dtype)
        pos = i32([p + k for _, p, n in part for k in range(n)], dev)
        qs = i32([0] + torch.tensor([n for *_, n in part]).cumsum(0).tolist(), dev)
        single = all(n == 1 for *_, n in part)
        y = ops.mingru(x, zb.to(dev), xb.to(dev), state, i32([(3, 1)[s] for s, *_ in part], dev), pos, qs, single)
        close(y, torch.cat([want[s][0][p:p + n] for s, p, n in part]), dtype, f"cut {cut}")
        for s, _, n in part:
            at[s] += n
    assert tuple(at) == lens
    close(state[3], want[0][1], F32)                               # the state is fp32 whatever the activations are
    close(state[1], want[1][1], F32)
    assert bool((state[0] == -3).all()) and bool((state[2] == -3).all())


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_padding_rows_leave_every_state_alone(dev, dtype):
    W, d = 20, 16
    st, cs = torch.full((2, W), 5.0, device=dev), torch.full((2, 3, d), 5.0, dtype=dtype, device=dev)
    args = (i32([-1, -1], dev), i32([0, 9], dev), i32([0, 1, 2], dev))
    ops.mingru(rnd(2, 3 * W).to(dev, dtype), rnd(W).to(dev), rnd(W).to(dev), st, *args, True)
    ops.mingru(rnd(2, 3 * W).to(dev, dtype), rnd(W).to(dev), rnd(W).to(dev), st, *args, False)
    ops.causal_conv(rnd(2, d).to(dev, dtype), rnd(4, d).to(dev), cs, *args)
    nxt = (torch.ones(d, device=dev), 1e-5, (rnd(4, d).to(dev), cs, args[0], args[1]))
    ops.embed_norm(rnd(9, d).to(dev, dtype), i32([3, 4], dev), torch.ones(d, device=dev), 1e-5, nxt)
    assert bool((st == 5).all()) and bool((cs == 5).all())


# ---- residual update, norms ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("d", [24, 1032, 2056, 5128, 8200])
@pytest.mark.parametrize("with_ff", [True, False])
def test_block_update_gates_sum_and_norm(dev, dtype, d, with_ff):
    T, k = 5, 3
    x, o, y = rnd(T, d, seed=1), rnd(T, d, seed=2), rnd(T * k, d, seed=3)
    g = rnd(T, 2 * d if with_ff else d, seed=4, scale=2.0)
    b1, b2, w = rnd(d, seed=5), rnd(d, seed=6), 1 + rnd(d, seed=7, scale=0.2)
    perm = torch.randperm(T * k, generator=torch.Generator().manual_seed(8)).view(T, k)
    wts = torch.rand(T, k, generator=torch.Generator().manual_seed(9))
    want = torch.sigmoid(g[:, :d] + b1) * o
    if with_ff:
        want = want + torch.sigmoid(g[:, d:] + b2) * (y[perm] * wts[..., None]).sum(1)
    want = x + 0.37 * want
    moe = (y.to(dev, dtype), perm.int().to(dev), wts.to(dev)) if with_ff else None
    xo, h, hc = ops.block_update(x.clone().to(dev), 0.37, o.to(dev, dtype), g.to(dev, dtype), b1.to(dev), b2.to(dev), moe, (w.to(dev), 1e-3, None))
    assert xo.dtype == F32 and hc is None
    close(xo, want, F32, "the residual stays fp32")
    close(h, O.norm_plain(want, w, 1e-3), dtype)
    xo, h, hc = ops.block_update(x.clone().to(dev), 0.37, o.to(dev, dtype), g.to(dev, dtype), b1.to(dev), b2.to(dev), moe, None)
    close(xo, want, F32)
    assert h is None


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("taps", [1, 2, 4])
def test_update_with_the_convolution_of_single_tokens(dev, dtype, taps):
    """Decode form: the convolution rides on the residual update; the same numbers as the separate launch, token after token,
    and a slot that starts over at position 0."""
    d, n = 40, 7
    table, w = rnd(30, d, seed=1), 1 + rnd(d, seed=2, scale=0.2)
    cw = rnd(taps, d, seed=3).to(dev)
    st = [torch.full((2, taps - 1, d), 9.0, dtype=dtype, device=dev) for _ in range(2)]
    for t in range(n):
        pos = i32([t % 5, t], dev)                                  # the first sequence starts over at t = 5
        slots, ids = i32([1, 0], dev), i32([3 * t % 30, t + 4], dev)
        nxt = (w.to(dev), 1e-5, (cw, st[0], slots, pos))
        x, h, hc = ops.embed_norm(table.to(dev, dtype), ids, w.to(dev), 1e-5, nxt)
        ref = ops.causal_conv(h, cw, st[1], slots, pos, i32([0, 1, 2], dev))
        assert torch.equal(hc, ref)
        assert torch.equal(st[0], st[1])
        want = O.norm_plain(table[ids.long().cpu()], w, 1e-5)
        close(x, want, F32)
        close(h, O.norm_plain(want, w, 1e-5), dtype)


@pytest.mark.parametrize("dev,dtype", WHERE)
def test_rms_rows_of_selected_rows(dev, dtype):
    x, w = rnd(9, 72, seed=1), rnd(72, seed=2)
    out = ops.rms_rows(x.to(dev), i32([8, 0, 8, 3], dev), w.to(dev), 0.5, dtype)
    close(out, O.norm_plain(x[[8, 0, 8, 3]], w, 0.5), dtype)


# ---- router ------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("E,k", [(5, 2), (3, 3), (64, 6), (4, 1)])
def test_router_bias_enters_choice_and_weights(dev, dtype, E, k):
    d, T = 64, 40
    h, w, b = rnd(T, d, seed=1), rnd(E, d, seed=2, scale=0.3), rnd(E, seed=3, scale=3.0)
    ids, wts = ops.moe_gate(h.to(dev, dtype), w.to(dev), None, k, 1, 1, 1.0, True, False, logit_bias=b.to(dev))
    ri, rw = O.router(h, {"router": w, "router.b": b}, "", {"router": {"top": k}})
    assert torch.equal(ids.long().cpu(), ri)
    close(wts, rw, F32)


# ---- expert products on CUDA cores ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("T", [1, 9, 150])
@pytest.mark.parametrize("d,F,E,k", [(48, 40, 5, 2), (40, 13, 3, 3), (64, 8, 4, 1)])
def test_expert_products(dev, dtype, T, d, F, E, k):
    x = rnd(T, d, seed=1)
    wg, wu, wd = rnd(E, F, d, seed=2, scale=0.2), rnd(E, F, d, seed=3, scale=0.2), rnd(E, d, F, seed=4, scale=0.3)
    g = torch.Generator().manual_seed(5)
    ids = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(T)]).int()
    put = lambda t: t.to(dev, dtype)                                # noqa: E731
    y, dest = ops.moe_routed(put(x), ids.to(dev), torch.ones(T, k, device=dev), put(wg), put(wu), put(wd))
    got = y.float().cpu()[dest.long().cpu()]                        # [T, k, d]
    a = torch.einsum("td,tkfd->tkf", x, wg[ids.long()])
    want = torch.einsum("tkf,tkdf->tkd", a * torch.sigmoid(a) * torch.einsum("td,tkfd->tkf", x, wu[ids.long()]), wd[ids.long()])
    close(got, want, dtype)


# ---- latent rows: norm, rotation, cache write ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("H,dn,dr,r", [(3, 24, 8, 40), (2, 10, 6, 15), (16, 128, 64, 512), (5, 7, 2, 9)])
@pytest.mark.parametrize("own_rows", [True, False])
def test_query_and_key_rotation_and_row_write(dev, dtype, H, dn, dr, r, own_rows):
    T, base, far = 6, 700.0, 5000
    q, ckv, w = rnd(T, H * (dn + dr), seed=1), rnd(T, r + dr, seed=2), 1 + rnd(r, seed=3, scale=0.2)
    pos = torch.tensor([0, 1, 2, 900, far, 3])
    table = ops.ref.yarn_table(far + 1, dr, base, 1.0, 0.0, 1.0, 0.0, 0.0, device=dev)
    slots = i32([4, 0, 7, -1, 9, 2], dev)
    both = torch.cat([q, ckv], 1).to(dev, dtype)
    cache = torch.full((11, r + dr), 5.0, dtype=dtype, device=dev)
    q_out = torch.zeros(T, H, r + dr, dtype=dtype, device=dev)
    qn = ops.mla_qkv_post(both[:, :q.shape[1]], both[:, q.shape[1]:] if own_rows else None, w.to(dev) if own_rows else None, 1e-3, table,
                          pos.int().to(dev), slots, cache, q_out, H, dn, dr, r, True)
    close(qn.reshape(T, H, dn), q.view(T, H, dn + dr)[..., :dn], F32)
    close(q_out[..., r:], O.rotate(q.view(T, H, dn + dr)[..., dn:].double(), pos, base, dr), dtype)
    if own_rows:
        want = torch.cat([O.norm_plain(ckv[:, :r], w, 1e-3), O.rotate(ckv[:, r:].double(), pos, base, dr).float()], 1)
        keep = [0, 1, 2, 4, 5]
        close(cache[[4, 0, 7, 9, 2]], want[keep], dtype)
        assert bool((cache[[1, 3, 5, 6, 8, 10]] == 5).all())
    else:
        assert bool((cache == 5).all())


# ---- windowed attention over paged rows ------------------------------------------------------------------------------------------------
def _paged(lens, row, dev, dtype, seed):
    """Rows of sequences scattered over blocks in random order: (cache, block tables, list of [S, row])."""
    bs, nb = 64, max((s + 63) // 64 for s in lens) + 1
    g = torch.Generator().manual_seed(seed)
    perm = torch.randperm(len(lens) * nb, generator=g).view(len(lens), nb)
    cache = torch.full((len(lens) * nb * bs, row), 50.0)             # rows nobody may see: a huge score, a huge value
    rows = []
    for b, S in enumerate(lens):
        x = (torch.randn(S, row, generator=g) * 0.5).bfloat16().float()
        rows.append(x)
        for p in range(S):
            cache[perm[b, p // bs] * bs + p % bs] = x[p]
    return cache, perm.int(), rows


def _attend(q, rows, r, scale, window):
    """q [n, H, D]: the last n positions of rows [S, D]."""
    n, S = q.shape[0], rows.shape[0]
    out = torch.zeros(n, q.shape[1], r)
    for k in range(n):
        i = S - n + k
        v = rows[max(0, i - window + 1):i + 1]
        out[k] = torch.softmax(q[k] @ v.T * scale, -1) @ v[:, :r]
    return out


SHAPES = [(3, 40, 8), (17, 15, 6), (1, 8, 2), (16, 512, 64), (5, 130, 16), (2, 700, 12)]


@pytest.mark.parametrize("dev,dtype", WHERE)
@pytest.mark.parametrize("H,r,dr", SHAPES)
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 130, 1000])
def test_windowed_attention_over_paged_rows(dev, dtype, H, r, dr, window):
    for lens, qlens in (([1, 70, 300, 129, 64], [1, 1, 1, 1, 1]), ([200, 66, 31], [73, 1, 31])):
        cache, bt, rows = _paged(lens, r + dr, dev, dtype, 3)
        T = sum(qlens)
        q = rnd(T, H, r + dr, seed=4, scale=0.3)
        qs = [0] + torch.tensor(qlens).cumsum(0).tolist()
        # the newest row inside the window and the first one outside it stand out for the last query of every sequence
        for b, (S, n) in enumerate(zip(lens, qlens)):
            i = S - 1
            for j in (i - window + 1, i - window):
                if 0 <= j < S:
                    v = (q[qs[b + 1] - 1, 0] * 1.5 + rnd(r + dr, seed=j, scale=0.5)).bfloat16().float()
                    rows[b][j] = v
                    cache[bt[b, j // 64].long() * 64 + j % 64] = v
        scale = 4.0 / (r + dr) ** 0.5
        want = torch.cat([_attend(q[a:e], x, r, scale, window) for x, a, e in zip(rows, qs, qs[1:])])
        got = ops.mla_attention(q.to(dev, dtype), cache.to(dev, dtype), bt.to(dev), i32(lens, dev), i32(qs, dev), scale, r, 64, max(qlens),
                                None, window)
        close(got, want, dtype, f"{lens} {qlens}")


@GPU
@pytest.mark.parametrize("window", [1, 64, 127, 128, 129, 300, 5000])
@pytest.mark.parametrize("lens,qlens", [([300], [300]), ([700], [130]), ([333, 90, 600], [200, 90, 1]), ([129, 1000], [129, 65])])
def test_windowed_prompt_attention_per_head(window, lens, qlens):
    """The tensor-core prompt kernel (per-head keys and values expanded from the visible rows only)."""
    nat, H, r, dn, dr, dv = ops.nat(), 4, 512, 128, 64, 128
    cache, bt, rows = _paged(lens, r + dr, "cuda", BF16, 5)
    T = sum(qlens)
    qs = [0] + torch.tensor(qlens).cumsum(0).tolist()
    q = rnd(T, H * (dn + dr), seed=6, scale=0.6)
    wkv = rnd(H, dn + dv, r, seed=7, scale=r ** -0.5)
    scale = 0.09
    meta = {"total_kv": sum(lens), "n_q_tiles": sum((n + 127) // 128 for n in qlens), "kv_decode": 0, "q_lens": qlens, "s_lens": lens}
    got = nat.mha_prefill(q.cuda().bfloat16(), cache.cuda().bfloat16(), wkv.reshape(-1, r).cuda().bfloat16(), bt.cuda(), i32(lens, "cuda"),
                          i32(qs, "cuda"), scale, H, 64, meta, window)
    nat.check_status()
    want = torch.zeros(T, H, dv)
    for x, a, e in zip(rows, qs, qs[1:]):
        kv = torch.einsum("sr,hdr->shd", x[:, :r], wkv)
        qq = q[a:e].view(e - a, H, dn + dr)
        s = (torch.einsum("nhd,shd->nhs", qq[..., :dn], kv[..., :dn]) + torch.einsum("nhd,sd->nhs", qq[..., dn:], x[:, r:])) * scale
        S, n = x.shape[0], e - a
        i, j = torch.arange(S - n, S)[:, None], torch.arange(S)[None]
        s = s.masked_fill(~((j <= i) & (i - j < window))[:, None], float("-inf"))
        want[a:e] = torch.einsum("nhs,shd->nhd", torch.softmax(s, -1), kv[..., dn:])
    close(got.view(T, H, dv), want, BF16)
