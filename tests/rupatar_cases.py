"""Small Rupatar configurations and random weights for the tests (no code of the package is used here)."""
import torch

from nibalix_cases import tokens, write_model  # noqa: F401  (the same for every folder model)


def attention(heads=6, kv_heads=2, dim=24, vdim=20, size=37, pool=5, rot=16, base=5000.0, factor=3.0, scale=0.3, v_mix=True, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix,
                                                       "mask": {"size": size, "pool": pool},
                                                       "rot": {"base": base, "dims": rot, "scaling": {"factor": factor}}}}


def hgrn2(heads=3, dim=20, vdim=24, mlp=None):
    return {"type": "hgrn2", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def mlstm(heads=3, dim=20, vdim=28, gate_cap=7.0, mlp=None):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}}


def moe(ff=24, experts=10, top=3, shared=24):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def config(layers, width=48, vocab=130, eps=1e-4, groups=3, scale=1.7):
    return {"architecture": "Rupatar", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "embedding": {"scale": scale}, "layers": layers}


CASES = {
    # every mixer, layers of different sizes and masks, one that mixes no values ahead of the first that does; shared experts as wide as one, two
    # and one and a half others, or none; a layer without a feed-forward
    "mixed": config([attention(v_mix=False, mlp=moe()), hgrn2(mlp=moe(ff=16, experts=7, top=2, shared=24)), attention(mlp=moe(shared=48)),
                     mlstm(), attention(heads=4, kv_heads=1, dim=16, vdim=40, size=20, pool=12, rot=16, factor=1.0, mlp=moe(top=1, shared=None)),
                     hgrn2(heads=4, dim=16, vdim=16), attention(heads=2, kv_heads=2, size=70, pool=9, mlp=moe(top=10))]),
    # sizes of one: heads, dimensions, window, pooled blocks, parts of the norm, experts
    "ones": config([attention(heads=1, kv_heads=1, dim=2, vdim=8, size=1, pool=1, rot=2, factor=1.0, mlp=moe(ff=8, experts=1, top=1, shared=8)),
                    hgrn2(heads=1, dim=1, vdim=1), mlstm(heads=1, dim=1, vdim=1, gate_cap=1.0, mlp=moe(ff=1, experts=2, top=1, shared=None)),
                    attention(heads=1, kv_heads=1, dim=8, vdim=8, size=3, pool=2, rot=8)], width=32, vocab=77, groups=1, scale=1.0),
    # sizes nothing divides, many query heads on one key head, a pooled block longer than a cache block, a width without 16-byte rows
    "odd": config([attention(heads=21, kv_heads=1, dim=13, vdim=9, size=23, pool=7, rot=6, mlp=moe(ff=19, experts=15, top=5, shared=7)), mlstm(heads=5, dim=11, vdim=7),
                   attention(heads=7, kv_heads=7, dim=6, vdim=9, size=11, pool=75, rot=0, v_mix=False), hgrn2(heads=7, dim=5, vdim=13, mlp=moe(ff=5, experts=3, top=3, shared=None))],
                  width=45, vocab=61, groups=9),
    # recurrences only, parts of eight columns
    "states": config([mlstm(heads=2, dim=40, vdim=16, gate_cap=15.0, mlp=moe(ff=40)), hgrn2(heads=2, dim=40, vdim=48), mlstm(heads=6, dim=8, vdim=8)], width=64, groups=8),
}


def weights(cfg, seed=0, dtype=torch.float32):
    """Tensor name -> tensor, written out from the configuration; matrices N(0, 1 / fan-in), rounded to bf16."""
    g = torch.Generator().manual_seed(seed)
    w = {}

    def mat(name, *shape, std=None, mean=0.0):
        w[name] = (mean + torch.randn(shape, generator=g) * (shape[-1] ** -0.5 if std is None else std)).bfloat16().to(dtype)

    d = cfg["width"]
    mat("embed", cfg["vocab"], d, std=0.6)
    for i, e in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", e["mixer"], e["mlp"]
        for k in ("norm1",) + (("norm2",) if f is not None else ()):
            mat(p + k, d, std=0.2, mean=1.0)
        p += "mix."
        H, n, v = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
        mat(p + "q", n, d)
        mat(p + "o", d, v)
        if e["type"] == "attention":
            G = m["kv_heads"]
            mat(p + "k", G * m["dim"], d)
            mat(p + "v", G * m["vdim"], d)
            mat(p + "g", v, d)
            for k, size in (("q", n), ("k", G * m["dim"]), ("v", G * m["vdim"]), ("o", d)):
                mat(p + k + ".b", size, std=0.3)
            if m["v_mix"]:
                mat(p + "vmix", std=0.2, mean=0.4)
        elif e["type"] == "hgrn2":
            mat(p + "f", n, d)
            mat(p + "f.b", n, std=1.5, mean=1.0)
            w[p + "lower"] = torch.rand(n, generator=g).mul(0.9).bfloat16().to(dtype)
            w[p + "lower"][::3] = 0
            mat(p + "v", v, d)
            mat(p + "norm", m["vdim"], std=0.2, mean=1.0)
        else:
            mat(p + "k", n, d)
            mat(p + "v", v, d)
            mat(p + "g", v, d)
            mat(p + "norm", v, std=0.2, mean=1.0)
            mat(p + "i", H, d, std=2 * d ** -0.5)
            mat(p + "i.b", H, std=2.0)
            mat(p + "f", H, d)
            mat(p + "f.b", H, std=1.0, mean=2.0)
        if f is not None:
            p = f"l{i}.mlp."
            parts = [(f"e{j}", f["expert"]["ff"]) for j in range(f["router"]["experts"])] + ([("shared", f["shared"]["ff"])] if "shared" in f else [])
            for name, ff in parts:
                mat(f"{p}{name}.up", ff, d)
                mat(f"{p}{name}.down", d, ff)
            mat(p + "router", f["router"]["experts"], d, std=2 * d ** -0.5)
    mat("final.norm", d, std=0.2, mean=1.0)
    mat("head", cfg["vocab"], d, std=4 * d ** -0.5)
    return w
