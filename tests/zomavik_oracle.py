"""A plain, slow Zomavik: one function per mechanism, whole sequences token by token, no cache, no batching.

``config`` is the parsed model configuration, ``w`` maps tensor names to tensors.  Nothing of the package is used here.
Everything runs in the dtype of the weights handed in (the tests use float32 or float64).
"""
import math

import torch


# ---- small functions ---------------------------------------------------------------------------------------------------------
def norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(x):
    return x / (1 + torch.exp(-x))


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0)


def short_conv(x, taps_w, bias):
    """x [n, ch], taps_w [ch, taps]: the last column meets the current row, rows before the first are zero; silu after it."""
    n, taps = x.shape[0], taps_w.shape[1]
    out = bias.expand(n, -1).clone()
    for t in range(n):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                out[t] = out[t] + taps_w[:, j] * x[src]
    return silu(out)


def capped(x, cap):
    return cap * torch.tanh(x / cap) if cap else x


# ---- attention -----------------------------------------------------------------------------------------------------------------
def rotate(v, rot):
    """v [n, heads, D] of positions 0 .. n - 1: element i turns with element i + dims / 2; elements from dims on stay."""
    half, pos = rot["dims"] // 2, torch.arange(v.shape[0]).double()
    out = v.clone()
    for i in range(half):
        a = pos * rot["base"] ** (-2.0 * i / rot["dims"])
        c, s = torch.cos(a).to(v.dtype)[:, None], torch.sin(a).to(v.dtype)[:, None]
        out[..., i] = v[..., i] * c - v[..., i + half] * s
        out[..., i + half] = v[..., i + half] * c + v[..., i] * s
    return out


def attend(q, k, v, scale, softcap, sink):
    """q [n, H, D], k [n, G, D], v [n, G, V] of one sequence from position 0, sink [H] -> [n, H, V]."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    future = torch.ones(n, n, dtype=torch.bool).triu(1)
    for h in range(H):
        s = capped((q[:, h] @ k[:, h // rep].T) * scale, softcap).masked_fill(future, -math.inf)
        top = torch.maximum(s.max(-1).values, sink[h])[:, None]
        e = torch.exp(s - top)
        out[:, h] = (e @ v[:, h // rep]) / (torch.exp(sink[h] - top) + e.sum(-1, keepdim=True))
    return out


def attention(h, w, p, m):
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (h @ w[p + c].T + w[p + c + ".b"] for c in "qkv")
    q, k = rotate(q.view(n, H, m["dim"]), m["rot"]), rotate(k.view(n, G, m["dim"]), m["rot"])
    o = attend(q, k, v.view(n, G, m["vdim"]), m["scale"], m.get("softcap"), w[p + "sink"])
    return o.reshape(n, H * m["vdim"]) @ w[p + "o"].T


# ---- selective scan ------------------------------------------------------------------------------------------------------------
def selective_scan(x, dt, A, B, C, D, s=None):
    """x, dt [n, ch], A [ch, N], B, C [n, N], D [ch]; S [ch, N] -> (y [n, ch], S)."""
    s = torch.zeros_like(A) if s is None else s.clone()
    out = []
    for t in range(x.shape[0]):
        s = torch.exp(dt[t][:, None] * A) * s + (dt[t] * x[t])[:, None] * B[t]
        out.append(s @ C[t] + D * x[t])
    return torch.stack(out), s


def mamba_inputs(h, w, p, m):
    """x, z, dt [n, inner], B, C [n, state]."""
    x, z = torch.split(h @ w[p + "in"].T, m["inner"], -1)
    x = short_conv(x, w[p + "conv"], w[p + "conv.b"])
    dt, B, C = torch.split(x @ w[p + "x"].T, [m["dt_rank"], m["state"], m["state"]], -1)
    return x, z, softplus(dt @ w[p + "dt"].T + w[p + "dt.b"]), B, C


def mamba(h, w, p, m):
    x, z, dt, B, C = mamba_inputs(h, w, p, m)
    y, _ = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), B, C, w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


def mixer(h, w, p, m):
    return m["left_scale"] * attention(h, w, p + "left.", m["left"]) + m["right_scale"] * mamba(h, w, p + "right.", m["right"])


# ---- feed-forward --------------------------------------------------------------------------------------------------------------
def dense(h, w, p):
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top, groups):
    """Router logits [n, E] -> weights [n, E], zero for the experts that are not chosen."""
    n, E = z.shape
    s = torch.exp(z - z.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    out = torch.zeros_like(s)
    size = E // groups["count"] if groups else E
    keep = groups["keep"] if groups else 1
    for t in range(n):
        best = sorted(range(E // size), key=lambda g: -float(s[t, g * size:(g + 1) * size].max()))[:keep]
        free = [e for g in best for e in range(g * size, (g + 1) * size)]
        pick = sorted(free, key=lambda e: (-float(s[t, e]), e))[:top]
        out[t, pick] = s[t, pick] / (s[t, pick].sum() + 1e-20)
    return out


def moe(h, w, p, m):
    r = m["router"]
    wt = route(h @ w[p + "router"].T, r["top"], r.get("groups"))
    out = torch.zeros_like(h)
    for e in range(wt.shape[1]):
        t = torch.nonzero(wt[:, e]).flatten()
        if t.numel():
            out[t] = out[t] + wt[t, e][:, None] * expert(h[t], w, p + f"e{e}.")
    if m.get("shared") is not None:
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * expert(h, w, p + "shared.")
    return out


# ---- the model -------------------------------------------------------------------------------------------------------------------
def layer(x, w, p, e, eps):
    y = x + mixer(norm(x, w[p + "norm1"], eps), w, p + "mix.", e["mixer"]) * w[p + "ls1"]
    if e.get("mlp") is None:
        return y
    h = norm(x, w[p + "norm2"], eps)
    return y + (dense(h, w, p + "mlp.") if e["mlp"]["kind"] == "dense" else moe(h, w, p + "mlp.", e["mlp"])) * w[p + "ls2"]


def order(config):
    """Layer indices in the order they run, and the places before which a pass of the loop starts."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n)), []
    a, b, times = loop["start"], loop["stop"], loop["times"]
    runs = list(range(a)) + [i for _ in range(times) for i in range(a, b)] + list(range(b, n))
    return runs, [a + k * (b - a) for k in range(times)]


def forward(config, w, tokens, layers_out=None):
    """Logits [n, vocab] of one sequence; ``layers_out`` (a list) collects the residual after every layer run."""
    eps = config["norm"]["eps"]
    x = x0 = w["embed"][torch.as_tensor(tokens).long()] * config["embedding"]["scale"]
    runs, starts = order(config)
    for k, i in enumerate(runs):
        if k in starts:
            x = torch.cat([x, x0], -1) @ w["loop.in"].T
        x = layer(x, w, f"l{i}.", config["layers"][i], eps)
        if layers_out is not None:
            layers_out.append(x)
    return capped(norm(x, w["final.norm"], eps) @ w["head"].T * config["logit_scale"], config.get("logit_softcap"))


def generate(config, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(config, w, toks)[-1])))
    return toks[len(prompt):]
