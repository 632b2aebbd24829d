"""A plain, slow Rupatar: one function per mechanism, whole sequences token by token, no cache, no batching.

``config`` is the parsed model configuration, ``w`` maps tensor names to tensors.  Nothing of the package is used here.
Everything runs in the dtype of the weights handed in (the tests use float32 or float64).
"""
import math

import torch


# ---- small functions ---------------------------------------------------------------------------------------------------------
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x, w, groups, eps):
    """Every one of ``groups`` equal parts of the row over its own root mean square."""
    parts = [rms(p, eps) for p in x.chunk(groups, -1)]
    return torch.cat(parts, -1) * w


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def log_sigmoid(x):
    return x.clamp_max(0) - torch.log1p(torch.exp(-x.abs()))


def gelu(x):
    return x * (1 + torch.erf(x / math.sqrt(2))) / 2


# ---- attention -----------------------------------------------------------------------------------------------------------------
def rotate(v, rot):
    """v [n, heads, D] of positions 0 .. n - 1: neighbours 2 i and 2 i + 1 turn together; elements from dims on stay."""
    n, stretch = v.shape[0], (rot.get("scaling") or {}).get("factor", 1.0)
    out, pos = v.clone(), torch.arange(n).double()
    for i in range(rot["dims"] // 2):
        a = pos * (rot["base"] ** (-2.0 * i / rot["dims"]) / stretch)
        c, s = torch.cos(a).to(v.dtype)[:, None], torch.sin(a).to(v.dtype)[:, None]
        out[..., 2 * i] = v[..., 2 * i] * c - v[..., 2 * i + 1] * s
        out[..., 2 * i + 1] = v[..., 2 * i + 1] * c + v[..., 2 * i] * s
    return out


def seen_tokens(i, size):
    """Positions a query at i sees one by one."""
    return list(range(max(0, i - size + 1), i + 1)) if size else list(range(i + 1))


def seen_blocks(i, size, pool):
    """Blocks a query at i sees as one key: their last token lies before the window."""
    return [b for b in range(i // pool + 1) if b * pool + pool - 1 <= i - size] if pool else []


def attend(q, k, v, scale, size, pool):
    """q [n, H, D], k [n, G, D], v [n, G, V] of one sequence from position 0 -> [n, H, V]; the softmax' denominator starts at one."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    full = n // pool if pool else 0
    mean = lambda x: torch.stack([x[b * pool:(b + 1) * pool].mean(0) for b in range(full)]) if full else x[:0]      # noqa: E731
    kb, vb = mean(k), mean(v)
    for i in range(n):
        t, b = seen_tokens(i, size), seen_blocks(i, size, pool)
        for h in range(H):
            keys = torch.cat([k[t, h // rep], kb[b, h // rep]])
            vals = torch.cat([v[t, h // rep], vb[b, h // rep]])
            s = (keys @ q[i, h]) * scale
            top = s.max().clamp_min(0)
            e = torch.exp(s - top)
            out[i, h] = (e @ vals) / (torch.exp(-top) + e.sum())
    return out


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


def attention(h, w, p, m, eps, first):
    """``first``: a list that holds the first mixing layer's values once there are any."""
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (h @ w[p + c].T + w[p + c + ".b"] for c in "qkv")
    q, k = (rms(rotate(x.view(n, -1, m["dim"]), m["rot"]), eps) for x in (q, k))
    if m.get("v_mix"):
        if first:
            v = mix_values(v, first[0], w[p + "vmix"])
        else:
            first.append(v)
    mask = m.get("mask") or {}
    o = attend(q, k, v.view(n, G, m["vdim"]), m["scale"], mask.get("size"), mask.get("pool"))
    return (o.reshape(n, H * m["vdim"]) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T + w[p + "o.b"]


# ---- recurrences ---------------------------------------------------------------------------------------------------------------
def hgrn2_scan(q, f, v, s=None):
    """q, f [n, H, K], v [n, H, V]; S [H, K, V] -> (o [n, H, V], S)."""
    s = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype) if s is None else s.clone()
    out = []
    for t in range(q.shape[0]):
        s = f[t][..., None] * s + (1 - f[t])[..., None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", s, q[t]))
    return torch.stack(out), s


def hgrn2(h, w, p, m, eps):
    n, H = h.shape[0], m["heads"]
    q, low = h @ w[p + "q"].T, w[p + "lower"]
    f = low + (1 - low) * sigmoid(h @ w[p + "f"].T + w[p + "f.b"])
    o, _ = hgrn2_scan((q * sigmoid(q)).view(n, H, -1), f.view(n, H, -1), (h @ w[p + "v"].T).view(n, H, -1))
    return (rms(o, eps) * w[p + "norm"]).reshape(n, -1) @ w[p + "o"].T


def mlstm_scan(q, k, v, i, f, state=None):
    """q, k [n, H, K], v [n, H, V], log gates i, f [n, H]; state (S [H, K, V], n [H, K], m [H])."""
    H, K, V = q.shape[1], q.shape[2], v.shape[2]
    S, nrm, top = (torch.zeros(H, K, V, dtype=q.dtype), torch.zeros(H, K, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)) if state is None else state
    out = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + top, i[t])
        keep, put = torch.exp(f[t] + top - new)[:, None], torch.exp(i[t] - new)[:, None]
        S = keep[..., None] * S + put[..., None] * k[t][:, :, None] * v[t][:, None, :]
        nrm, top = keep * nrm + put * k[t], new
        size = torch.maximum((nrm * q[t]).sum(-1).abs(), torch.exp(-top)) + 1e-6
        out.append(torch.einsum("hkv,hk->hv", S, q[t]) / size[:, None])
    return torch.stack(out), (S, nrm, top)


def mlstm(h, w, p, m, eps):
    n, H, K, cap = h.shape[0], m["heads"], m["dim"], m["gate_cap"]
    q, k, v = ((h @ w[p + c].T).view(n, H, -1) for c in "qkv")
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o, _ = mlstm_scan(q * K ** -0.5, k, v, i, f)
    return (rms(o, eps).reshape(n, -1) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- feed-forward --------------------------------------------------------------------------------------------------------------
def expert(h, w, p):
    return gelu(h @ w[p + "up"].T) @ w[p + "down"].T


def route(z, top):
    """Router logits [n, E] -> weights [n, E], zero for the experts that are not chosen."""
    s = sigmoid(z)
    out = torch.zeros_like(s)
    for t in range(z.shape[0]):
        pick = sorted(range(z.shape[1]), key=lambda e: (-float(s[t, e]), e))[:top]        # noqa: B023
        out[t, pick] = s[t, pick]
    return out


def moe(h, w, p, m):
    wt = route(h @ w[p + "router"].T, m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(wt.shape[1]):
        t = torch.nonzero(wt[:, e]).flatten()
        if t.numel():
            out[t] = out[t] + expert(wt[t, e][:, None] * h[t], w, p + f"e{e}.")
    return out + expert(h, w, p + "shared.") if m.get("shared") is not None else out


# ---- the model -------------------------------------------------------------------------------------------------------------------
def layer(x, w, p, e, norm, first):
    eps, m = norm["eps"], e["mixer"]
    h = group_norm(x, w[p + "norm1"], norm["groups"], eps)
    x = x + (attention(h, w, p + "mix.", m, eps, first) if e["type"] == "attention" else {"hgrn2": hgrn2, "mlstm": mlstm}[e["type"]](h, w, p + "mix.", m, eps))
    if e.get("mlp") is None:
        return x
    return x + moe(group_norm(x, w[p + "norm2"], norm["groups"], eps), w, p + "mlp.", e["mlp"])


def forward(config, w, tokens, layers_out=None):
    """Logits [n, vocab] of one sequence; ``layers_out`` (a list) collects the residual after every layer."""
    norm, first = config["norm"], []
    x = w["embed"][torch.as_tensor(tokens).long()] * config["embedding"]["scale"]
    for i, e in enumerate(config["layers"]):
        x = layer(x, w, f"l{i}.", e, norm, first)
        if layers_out is not None:
            layers_out.append(x)
    return group_norm(x, w["final.norm"], norm["groups"], norm["eps"]) @ w["head"].T


def generate(config, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(config, w, toks)[-1])))
    return toks[len(prompt):]
