"""A plain, slow Lugovik: one function per mechanism, whole sequences token by token, no cache, no batching.

``config`` is the parsed model configuration, ``w`` maps tensor names to tensors.  Nothing of the package is used here.
Everything runs in the dtype of the weights handed in (the tests use float32 or float64).
"""
import math

import torch


# ---- small functions ---------------------------------------------------------------------------------------------------------
def norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0)


def gelu_tanh(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def short_conv(x, taps_w, bias=None):
    """x [n, ch], taps_w [ch, taps]: the last column meets the current row, rows before the first are zero; silu after it."""
    n, taps = x.shape[0], taps_w.shape[1]
    out = torch.zeros_like(x)
    for t in range(n):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                out[t] += taps_w[:, j] * x[src]
    return silu(out if bias is None else out + bias)


# ---- rotation ------------------------------------------------------------------------------------------------------------------
def frequencies(dims, base, scaling):
    """Angle per position of every pair, and the factor on cos and sin."""
    f, mult = [base ** (-2.0 * i / dims) for i in range(dims // 2)], 1.0
    if scaling is not None:
        turn = lambda t: dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))       # noqa: E731
        lo, hi = max(math.floor(turn(scaling["fast"])), 0), min(math.ceil(turn(scaling["slow"])), dims - 1)
        for i in range(dims // 2):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f[i] = f[i] / scaling["factor"] * ramp + f[i] * (1 - ramp)
        mult = 0.1 * math.log(scaling["factor"]) + 1
    return f, mult


def rotate(v, pos, rot):
    """v [n, heads, D]: element i turns with element i + dims / 2; elements from dims on stay."""
    half = rot["dims"] // 2
    f, mult = frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    out = v.clone()
    for i in range(half):
        a = pos.double() * f[i]
        c, s = (torch.cos(a) * mult).to(v.dtype)[:, None], (torch.sin(a) * mult).to(v.dtype)[:, None]
        out[..., i] = v[..., i] * c - v[..., i + half] * s
        out[..., i + half] = v[..., i + half] * c + v[..., i] * s
    return out


# ---- attention -----------------------------------------------------------------------------------------------------------------
def attend(q, k, v, scale, softcap, chunk):
    """q [n, H, D], k [n, G, D], v [n, G, V] of one sequence from position 0 -> [n, H, V]."""
    n, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for i in range(n):
        lo = i // chunk * chunk
        for h in range(H):
            s = (k[lo:i + 1, h // rep] @ q[i, h]) * scale
            e = torch.exp(softcap * torch.tanh(s / softcap))
            out[i, h] = (e @ v[lo:i + 1, h // rep]) / (1 + e.sum())
    return out


def gated_attention(h, w, p, m, eps):
    n, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(n)
    q = rotate(norm((h @ w[p + "q"].T).view(n, H, D), w[p + "q.norm"], eps), pos, m["rot"])
    k = rotate(norm((h @ w[p + "k"].T).view(n, G, D), w[p + "k.norm"], eps), pos, m["rot"])
    v = (h @ w[p + "v"].T).view(n, G, V)
    o = attend(q, k, v, m["scale"], m["softcap"], m["mask"]["size"])
    o = o * torch.sigmoid(h @ w[p + "g"].T)[..., None]
    return o.reshape(n, H * V) @ w[p + "o"].T


# ---- recurrences: S [heads, key channels, value channels] ------------------------------------------------------------------------
def linear_state(q, k, v, decay, s=None):
    """S_t = diag(decay_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t; q, k, decay [n, H, K], v [n, H, V]."""
    n, H, K = q.shape
    s = torch.zeros(H, K, v.shape[2], dtype=q.dtype) if s is None else s.clone()
    out = []
    for t in range(n):
        s = decay[t][..., None] * s + k[t][..., None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", s, q[t]))
    return torch.stack(out), s


def delta_state(q, k, v, decay, beta, s=None):
    """S <- diag(decay) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    n, H, K = q.shape
    s = torch.zeros(H, K, v.shape[2], dtype=q.dtype) if s is None else s.clone()
    out = []
    for t in range(n):
        s = decay[t][..., None] * s
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", s, k[t]))
        s = s + k[t][..., None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", s, q[t]))
    return torch.stack(out), s


def channel_delta_inputs(h, w, p, m):
    """q, k [n, H, K], v [n, H, V], decay [n, H, K], beta [n, H]."""
    n, H, G, K, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).view(n, G, K)) * K ** -0.5
    k = unit(short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).view(n, G, K))
    v = short_conv(h @ w[p + "v"].T, w[p + "v.conv"]).view(n, H, V)
    head = torch.arange(H) // (H // G)
    sp = softplus((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(n, H, K)
    decay = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * sp)
    return q[:, head], k[:, head], v, decay, torch.sigmoid(h @ w[p + "b"].T)


def channel_delta(h, w, p, m, eps):
    n, H, V = h.shape[0], m["heads"], m["vdim"]
    o, _ = delta_state(*channel_delta_inputs(h, w, p, m))
    o = norm(o, w[p + "norm"], eps) * torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(n, H, V)
    return o.reshape(n, H * V) @ w[p + "o"].T


def gated_linear(h, w, p, m, eps):
    n, H, K, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = (h @ w[p + "q"].T).view(n, H, K) * K ** -0.5, (h @ w[p + "k"].T).view(n, H, K)
    v = (h @ w[p + "v"].T).view(n, H, V)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
    alpha = torch.exp(-softplus(-z) / m["tau"]).view(n, H, K)
    o, _ = linear_state(q, k, v, alpha)
    o = norm(o, w[p + "norm"], eps).reshape(n, H * V) * silu(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def mamba2(h, w, p, m, eps):
    n, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], -1)
    x, B, C = torch.split(short_conv(xbc, w[p + "conv"], w[p + "conv.b"]), [inner, G * N, G * N], -1)
    group = torch.arange(H) // (H // G)
    x, B, C = x.view(n, H, V), B.view(n, G, N)[:, group], C.view(n, G, N)[:, group]
    dt = softplus(dt + w[p + "dt_bias"])
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * dt)[..., None].expand(n, H, N)
    y, _ = linear_state(C, B, dt[..., None] * x, decay)
    y = (y + w[p + "D"][None, :, None] * x).reshape(n, inner) * silu(z)
    ng = m["norm_groups"]
    y = norm(y.view(n, ng, inner // ng), w[p + "norm"].view(ng, inner // ng), eps).reshape(n, inner)
    return y @ w[p + "o"].T


# ---- the model -------------------------------------------------------------------------------------------------------------------
def mixer(h, w, p, layer, eps):
    m = layer["mixer"]
    if layer["type"] == "mamba2":
        return mamba2(h, w, p, m, eps)
    if layer["type"] == "channel_delta":
        return channel_delta(h, w, p, m, eps)
    return m["left_scale"] * gated_attention(h, w, p + "left.", m["left"], eps) + \
        m["right_scale"] * gated_linear(h, w, p + "right.", m["right"], eps)


def feed_forward(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(config, w, tokens, layers_out=None):
    """Logits [n, vocab] of one sequence; ``layers_out`` (a list) collects the residual after every layer."""
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens).long()] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + norm(mixer(norm(x, w[p + "norm1"], eps), w, p + "mix.", layer, eps), w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            x = x + norm(feed_forward(norm(x, w[p + "norm2"], eps), w, p + "mlp."), w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, w["final.norm"], eps) @ w["head"].T


def generate(config, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(forward(config, w, toks)[-1])))
    return toks[len(prompt):]
