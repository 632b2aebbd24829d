"""A plain, slow Nibalix: one function per mechanism, whole sequences at once, no cache, no batching.

``config`` is the parsed model configuration, ``w`` maps tensor names to tensors.  Nothing of the package is used here.
Everything runs in the dtype of the weights handed in (the tests use float32 or float64).
"""
import math

import torch


def rms(x, eps):
    """Root mean square with eps under the root."""
    return torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_one(x, w, eps):
    """The stored weight is the deviation from one."""
    return x / rms(x, eps) * (1 + w)


def norm_plain(x, w, eps):
    return x / rms(x, eps) * w


def rotate(v, pos, base, dims):
    """v [n, ..., D]: element i < dims / 2 turns with element i + dims / 2 by pos * base^(-2 i / dims)."""
    half = dims // 2
    out = v.clone()
    for i in range(half):
        ang = pos.double() * base ** (-2.0 * i / dims)
        c, s = torch.cos(ang).to(v.dtype), torch.sin(ang).to(v.dtype)
        shape = [-1] + [1] * (v.dim() - 2)
        c, s = c.view(shape), s.view(shape)
        out[..., i] = v[..., i] * c - v[..., i + half] * s
        out[..., i + half] = v[..., i + half] * c + v[..., i] * s
    return out


def input_conv(h, taps_w):
    """h [n, d], taps_w [d, taps]: the last tap meets the current row; rows before the first are zero."""
    n, d = h.shape
    taps = taps_w.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, d, dtype=h.dtype), h], 0)
    out = torch.zeros_like(h)
    for j in range(taps):
        out += taps_w[:, j] * pad[j:j + n]
    return out


def latent_rows(h, w, p, m, eps):
    """(normed latent, rotated shared key part) of every token."""
    r = m["kv_rank"]
    y = h @ w[p + "dkv"].T
    c = norm_plain(y[:, :r], w[p + "dkv.norm"], eps)
    k = rotate(y[:, r:], torch.arange(h.shape[0]), m["rot"]["base"], m["rot"]["dims"])
    return c, k


def latent_attention(h, rows, w, p, m):
    """Windowed softmax attention in the expanded per-head form."""
    n, H = h.shape[0], m["heads"]
    dn, dr, dv = m["dim"], m["rot_dim"], m["vdim"]
    c, kr = rows
    q = (h @ w[p + "q"].T).view(n, H, dn + dr)
    qn, qr = q[..., :dn], rotate(q[..., dn:], torch.arange(n), m["rot"]["base"], m["rot"]["dims"])
    kn = (c @ w[p + "uk"].T).view(n, H, dn)
    v = (c @ w[p + "uv"].T).view(n, H, dv)
    out = torch.zeros(n, H, dv, dtype=h.dtype)
    for i in range(n):
        lo = max(0, i - m["mask"]["size"] + 1)
        s = (torch.einsum("hd,jhd->hj", qn[i], kn[lo:i + 1]) + torch.einsum("hd,jd->hj", qr[i], kr[lo:i + 1])) * m["scale"]
        out[i] = torch.einsum("hj,jhd->hd", torch.softmax(s, -1), v[lo:i + 1])
    return out.reshape(n, H * dv) @ w[p + "o"].T


def mingru(h, w, p):
    z = torch.sigmoid(h @ w[p + "z"].T + w[p + "z.b"])
    u = h @ w[p + "x"].T + w[p + "x.b"]
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    g = h @ w[p + "g"].T
    s = torch.zeros_like(z[0])
    ys = []
    for t in range(h.shape[0]):
        s = (1 - z[t]) * s + z[t] * cand[t]
        ys.append(s * (g[t] * torch.sigmoid(g[t])))
    return torch.stack(ys) @ w[p + "o"].T


def router(h, w, p, m):
    """Chosen experts and their weights, per token."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    v, i = torch.topk(z, m["router"]["top"], dim=-1)
    return i, torch.softmax(v, -1)


def experts(h, w, p, m):
    ids, wt = router(h, w, p, m)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k in range(ids.shape[1]):
            e = p + f"e{int(ids[t, k])}."
            a = w[e + "gate"] @ h[t]
            out[t] += wt[t, k] * (w[e + "down"] @ (a * torch.sigmoid(a) * (w[e + "up"] @ h[t])))
    return out


def gate(h, w, name):
    return torch.sigmoid(h @ w[name].T + w[name + ".b"])


def forward(config, w, tokens, layers_out=None):
    """Logits [n, vocab] of one sequence; ``layers_out`` (a list) collects the residual after every layer."""
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = norm_around_one(w["embed"][torch.as_tensor(tokens).long()], w["embed.norm"], eps)
    rows = {}
    for i, layer in enumerate(config["layers"]):
        p, mix = f"l{i}.", layer["mixer"]
        h = norm_around_one(x, w[p + "norm1"], eps)
        hm = h + input_conv(h, w[p + "canon1"])
        if layer["type"] == "mingru":
            y = mingru(hm, w, p + "mix.")
        else:
            src = mix.get("kv_from")
            if src is None:
                rows[i] = latent_rows(hm, w, p + "mix.", mix, eps)
            y = latent_attention(hm, rows[i if src is None else src], w, p + "mix.", mix)
        y = gate(h, w, p + "rg1") * y
        if layer.get("mlp") is not None:
            y = y + gate(h, w, p + "rg2") * experts(h, w, p + "mlp.", layer["mlp"])
        x = x + m * y
        if layers_out is not None:
            layers_out.append(x)
    return norm_around_one(x, w["final.norm"], eps) @ w["head"].T


def generate(config, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(config, w, toks)[-1])))
    return toks[len(prompt):]
