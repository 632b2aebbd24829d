"""Small Lugovik configurations and random weights for the tests (no code of the package is used here)."""
import torch

from nibalix_cases import tokens, write_model  # noqa: F401  (the same for every folder model)


def mamba(heads=3, vdim=20, state=24, groups=1, norm_groups=1, conv=3):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def delta(heads=4, kv_heads=2, dim=20, vdim=28, conv=4):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def parallel(heads=6, kv_heads=2, dim=24, vdim=20, chunk=50, rot=16, base=5000.0, scaling=(3.0, 96, 8.0, 1.0), scale=0.21, softcap=11.0, rheads=3, rdim=12,
             rvdim=20, tau=9.0, left=0.7, right=1.3):
    r = {"base": base, "dims": rot}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "rot": r, "scale": scale, "softcap": softcap},
        "left_scale": left, "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "tau": tau}, "right_scale": right}}


def config(layers, width=48, vocab=130, eps=1e-4, scale=3.1, ff=72):
    out = []
    for e in layers:
        e = dict(e)
        e.setdefault("mlp", {"kind": "dense", "ff": ff} if ff else None)
        out.append(e)
    return {"architecture": "Lugovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": out}


CASES = {
    # every mechanism, layers of different sizes and orders, one without a feed-forward
    "mixed": config([parallel(), mamba(heads=6, groups=2, norm_groups=3, conv=2), dict(delta(), mlp=None), mamba(),
                     parallel(heads=4, kv_heads=4, dim=16, vdim=32, chunk=64, rot=16, softcap=40.0, scaling=(2.0, 64, 32.0, 2.0), rheads=2, rdim=40, rvdim=12),
                     dict(delta(heads=3, kv_heads=3, dim=36, vdim=16, conv=3), mlp={"kind": "dense", "ff": 40})]),
    # sizes of one, no short convolution to speak of, one query head, chunks of three tokens
    "ones": config([delta(heads=1, kv_heads=1, dim=8, vdim=4, conv=1), mamba(heads=1, vdim=8, state=1, conv=1),
                    parallel(heads=1, kv_heads=1, dim=8, vdim=8, chunk=3, rot=2, rheads=1, rdim=8, rvdim=8, tau=1.0, left=1.0, right=1.0)],
                   width=32, vocab=77, ff=8),
    # sizes nothing divides, deep convolutions, many query heads on one key head, a width without 16-byte rows, no scaling
    "odd": config([delta(heads=6, kv_heads=2, dim=11, vdim=7, conv=6), parallel(heads=21, kv_heads=1, dim=13, vdim=9, chunk=37, rot=6, scaling=None, rheads=5,
                                                                            rdim=3, rvdim=5), mamba(heads=9, vdim=5, state=7, groups=3, norm_groups=5, conv=7)],
                  width=43, vocab=61, ff=29),
    # the recurrences alone: no layer has paged rows
    "states": config([mamba(heads=2, vdim=36, state=16, groups=2, norm_groups=2, conv=5), delta(heads=2, kv_heads=1, dim=48, vdim=8)], width=40, ff=None),
}


def weights(cfg, seed=0, dtype=torch.float32, rank=10):
    """Tensor name -> tensor, written out from the configuration; matrices N(0, 1 / fan-in), rounded to bf16."""
    g = torch.Generator().manual_seed(seed)
    w = {}

    def mat(name, *shape, std=None, mean=0.0):
        w[name] = (mean + torch.randn(shape, generator=g) * (shape[-1] ** -0.5 if std is None else std)).bfloat16().to(dtype)

    d = cfg["width"]
    norm = lambda name, n: mat(name, n, std=0.2, mean=1.0)           # noqa: E731
    mat("embed", cfg["vocab"], d, std=0.4)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        for k in ("norm1", "norm1b") + (("norm2", "norm2b") if e["mlp"] is not None else ()):
            norm(p + k, d)
        if e["mlp"] is not None:
            ff = e["mlp"]["ff"]
            mat(p + "mlp.gate", ff, d)
            mat(p + "mlp.up", ff, d)
            mat(p + "mlp.down", d, ff)
        p += "mix."
        if e["type"] == "mamba2":
            inner, gn, H = m["heads"] * m["vdim"], m["groups"] * m["state"], m["heads"]
            mat(p + "in", 2 * inner + 2 * gn + H, d)
            mat(p + "conv", inner + 2 * gn, m["conv"], std=0.6)
            mat(p + "conv.b", inner + 2 * gn, std=0.3)
            mat(p + "dt_bias", H, std=1.0, mean=-2.0)
            mat(p + "A_log", H, std=0.7)
            mat(p + "D", H, std=1.0)
            norm(p + "norm", inner)
            mat(p + "o", d, inner)
        elif e["type"] == "channel_delta":
            H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for k, n in (("q", G * K), ("k", G * K), ("v", H * V)):
                mat(p + k, n, d)
                mat(p + k + ".conv", n, m["conv"], std=0.6)
            mat(p + "b", H, d)
            mat(p + "A_log", H, std=0.7)
            norm(p + "norm", V)
            mat(p + "a1", rank, d)
            mat(p + "a2", H * K, rank)
            mat(p + "dt_bias", H * K, std=1.5, mean=-3.0)
            mat(p + "g1", rank + 3, d)
            mat(p + "g2", H * V, rank + 3)
            mat(p + "o", d, H * V)
        else:
            a, r = m["left"], m["right"]
            q = p + "left."
            mat(q + "q", a["heads"] * a["dim"], d)
            mat(q + "k", a["kv_heads"] * a["dim"], d)
            mat(q + "v", a["kv_heads"] * a["vdim"], d)
            norm(q + "q.norm", a["dim"])
            norm(q + "k.norm", a["dim"])
            mat(q + "g", a["heads"], d, std=1.5 * d ** -0.5)
            mat(q + "o", d, a["heads"] * a["vdim"])
            q = p + "right."
            mat(q + "q", r["heads"] * r["dim"], d)
            mat(q + "k", r["heads"] * r["dim"], d)
            mat(q + "v", r["heads"] * r["vdim"], d)
            mat(q + "g", r["heads"] * r["vdim"], d)
            mat(q + "o", d, r["heads"] * r["vdim"])
            norm(q + "norm", r["vdim"])
            mat(q + "a1", rank - 1, d)
            mat(q + "a2", r["heads"] * r["dim"], rank - 1)
            mat(q + "a2.b", r["heads"] * r["dim"], std=1.5)
    norm("final.norm", d)
    mat("head", cfg["vocab"], d)
    return w
