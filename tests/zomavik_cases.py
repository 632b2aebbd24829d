"""Small Zomavik configurations and random weights for the tests (no code of the package is used here)."""
import torch

from nibalix_cases import tokens, write_model  # noqa: F401  (the same for every folder model)


def layer(heads=6, kv_heads=2, dim=24, vdim=20, rot=16, base=5000.0, scale=0.21, softcap=11.0, inner=40, state=12, dt_rank=5, conv=4, left=0.7,
          right=1.3, mlp=None):
    left_part = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot}, "scale": scale, "softcap": softcap}
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": left_part, "left_scale": left, "right_scale": right,
                                                      "right": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=12, top=3, groups=(3, 2), shared=24):
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": r}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def config(layers, width=48, vocab=130, eps=1e-4, scale=1.7, loop=None, logit_scale=0.6, logit_softcap=9.0):
    c = {"architecture": "Zomavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers,
         "logit_scale": logit_scale, "logit_softcap": logit_softcap}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CASES = {
    # every feed-forward, layers of different sizes, a loop in the middle; shared experts as wide as one, two and one and a half others
    "mixed": config([layer(mlp=dense()), layer(mlp=moe()), layer(heads=4, kv_heads=4, dim=16, vdim=32, rot=16, inner=64, state=16, dt_rank=8, conv=3),
                     layer(mlp=moe(ff=16, experts=10, top=4, groups=None, shared=24), softcap=30.0), layer(mlp=moe(shared=48, groups=(4, 1)), conv=2)],
                    loop=(1, 3, 2)),
    # sizes of one: heads, taps, state, rank, passes, experts; the loop covers the whole model
    "ones": config([layer(heads=1, kv_heads=1, dim=8, vdim=8, rot=2, inner=8, state=1, dt_rank=1, conv=1, left=1.0, right=1.0,
                          mlp=moe(ff=8, experts=1, top=1, groups=None, shared=8)), layer(heads=1, kv_heads=1, dim=2, vdim=1, rot=2, inner=1, mlp=dense(1))],
                   width=32, vocab=77, loop=(0, 2, 1), logit_scale=1.0),
    # sizes nothing divides, deep convolutions, many query heads on one key head, a width without 16-byte rows; the loop begins at once
    "odd": config([layer(heads=21, kv_heads=1, dim=13, vdim=9, rot=6, inner=37, state=23, dt_rank=11, conv=7, mlp=moe(ff=19, experts=15, top=5, groups=(5, 3), shared=7)),
                   layer(heads=6, kv_heads=3, dim=11, vdim=7, rot=4, inner=51, state=3, dt_rank=2, conv=5, mlp=dense(29))],
                  width=43, vocab=61, loop=(0, 1, 3)),
    # no loop, no softcaps, no shared expert, no groups
    "plain": config([layer(softcap=None, mlp=moe(ff=40, experts=6, top=2, groups=None, shared=None)), layer(state=40, inner=24, softcap=None)],
                    logit_scale=1.0, logit_softcap=None),
}


def weights(cfg, seed=0, dtype=torch.float32):
    """Tensor name -> tensor, written out from the configuration; matrices N(0, 1 / fan-in), rounded to bf16."""
    g = torch.Generator().manual_seed(seed)
    w = {}

    def mat(name, *shape, std=None, mean=0.0):
        w[name] = (mean + torch.randn(shape, generator=g) * (shape[-1] ** -0.5 if std is None else std)).bfloat16().to(dtype)

    d = cfg["width"]
    mat("embed", cfg["vocab"], d, std=0.6)
    if cfg.get("loop"):
        mat("loop.in", d, 2 * d)
    for i, e in enumerate(cfg["layers"]):
        p, a, r, m = f"l{i}.", e["mixer"]["left"], e["mixer"]["right"], e["mlp"]
        for k in ("norm1", "ls1") + (("norm2", "ls2") if m is not None else ()):
            mat(p + k, d, std=0.2, mean=1.0)
        q = p + "mix.left."
        for k, n in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
            mat(q + k, n, d)
            mat(q + k + ".b", n, std=0.4)
        mat(q + "sink", a["heads"], std=1.5)
        mat(q + "o", d, a["heads"] * a["vdim"])
        q = p + "mix.right."
        inner, N, R = r["inner"], r["state"], r["dt_rank"]
        mat(q + "in", 2 * inner, d)
        mat(q + "conv", inner, r["conv"], std=0.6)
        mat(q + "conv.b", inner, std=0.3)
        mat(q + "x", R + 2 * N, inner, std=1.5 * inner ** -0.5)
        mat(q + "dt", inner, R)
        mat(q + "dt.b", inner, std=1.0, mean=-2.0)
        mat(q + "A_log", inner, N, std=0.7)
        mat(q + "D", inner, std=1.0)
        mat(q + "o", d, inner)
        p += "mlp."
        if m is not None and m["kind"] == "dense":
            mat(p + "up", m["ff"], d)
            mat(p + "down", d, m["ff"])
        elif m is not None:
            parts = [(f"e{j}", m["expert"]["ff"]) for j in range(m["router"]["experts"])] + ([("shared", m["shared"]["ff"])] if "shared" in m else [])
            for name, ff in parts:
                mat(f"{p}{name}.gate", ff, d)
                mat(f"{p}{name}.up", ff, d)
                mat(f"{p}{name}.down", d, ff)
            mat(p + "router", m["router"]["experts"], d, std=2 * d ** -0.5)
            if "shared" in m:
                mat(p + "shared.sg", 1, d)
    mat("final.norm", d, std=0.2, mean=1.0)
    mat("head", cfg["vocab"], d, std=4 * d ** -0.5)
    return w
