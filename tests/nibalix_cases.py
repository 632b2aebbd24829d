"""Small Nibalix configurations and random weights for the tests (no code of the package is used here)."""
import json
import os
import struct

import torch


def latent(heads=3, dim=24, rot=8, vdim=16, rank=40, window=37, base=5000.0, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale or (dim + rot) ** -0.5,
         "mask": {"size": window}, "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def gru(width=72):
    return {"type": "mingru", "mixer": {"width": width}}


def moe(ff=40, experts=5, top=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(layers, width=48, vocab=130, taps=4, eps=1e-4, mult=0.4, mlp="default"):
    out = []
    for e in layers:
        e = dict(e)
        e.setdefault("mlp", moe() if mlp == "default" else mlp)
        out.append(e)
    return {"architecture": "Nibalix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "canon": {"taps": taps}, "layers": out}


CASES = {
    # every mechanism, layers of different sizes, a source that two layers read, one of them with other head counts
    "mixed": config([gru(72), latent(), latent(heads=5, window=70, base=900.0, rank=24),
                     dict(latent(heads=2, vdim=40, dim=16, rank=24, window=11, base=900.0, kv_from=2), mlp=None), dict(gru(33), mlp=moe(24, 3, 3)),
                     latent(heads=17, rank=24, base=900.0, dim=8, window=70, kv_from=2)]),
    # attention only; one tap (no convolution state), one expert, a window of one
    "ones": config([latent(window=1, heads=1), latent(rank=8, rot=2, window=200, kv_from=None)], taps=1, width=32, vocab=77, mlp=moe(8, 4, 1)),
    # recurrence only, two taps, no feed-forward
    "gru": config([gru(16), gru(40)], taps=2, width=64, mlp=None),
    # rows of odd byte counts (nothing the tensor-core copies could address), deep convolution, all experts chosen
    "odd": config([latent(heads=3, dim=10, rot=6, vdim=9, rank=15, window=23), gru(25)], width=40, vocab=61, taps=7, mlp=moe(13, 2, 2)),
}


def weights(cfg, seed=0, dtype=torch.float32):
    """Tensor name -> tensor, written out from the configuration; matrices N(0, 1 / fan-in), rounded to bf16."""
    g = torch.Generator().manual_seed(seed)
    w = {}

    def mat(name, *shape, std=None):
        w[name] = (torch.randn(shape, generator=g) * (shape[-1] ** -0.5 if std is None else std)).bfloat16().to(dtype)

    d = cfg["width"]
    mat("embed", cfg["vocab"], d, std=1.0)
    mat("embed.norm", d, std=0.2)
    for i, e in enumerate(cfg["layers"]):
        p, m = f"l{i}.", e["mixer"]
        mat(p + "norm1", d, std=0.2)
        if e["type"] == "latent_attention":
            mat(p + "mix.q", m["heads"] * (m["dim"] + m["rot_dim"]), d)
            if "kv_from" not in m:
                mat(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], d)
                mat(p + "mix.dkv.norm", m["kv_rank"], std=0.2)
                w[p + "mix.dkv.norm"] += 1
                w[p + "mix.dkv.norm"] = w[p + "mix.dkv.norm"].bfloat16().to(dtype)
            mat(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"])
            mat(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
            mat(p + "mix.o", d, m["heads"] * m["vdim"])
        else:
            for k in ("z", "x"):
                mat(p + f"mix.{k}", m["width"], d)
                mat(p + f"mix.{k}.b", m["width"], std=0.5)
            mat(p + "mix.g", m["width"], d)
            mat(p + "mix.o", d, m["width"])
        if e["mlp"] is not None:
            ff, E = e["mlp"]["expert"]["ff"], e["mlp"]["router"]["experts"]
            for x in range(E):
                mat(p + f"mlp.e{x}.gate", ff, d)
                mat(p + f"mlp.e{x}.up", ff, d)
                mat(p + f"mlp.e{x}.down", d, ff)
            mat(p + "mlp.router", E, d, std=2 * d ** -0.5)
            mat(p + "mlp.router.b", E, std=1.0)
        mat(p + "canon1", d, cfg["canon"]["taps"], std=0.4)
        for k in ("rg1", "rg2") if e["mlp"] is not None else ("rg1",):
            mat(p + k, d, d)
            mat(p + k + ".b", d, std=0.5)
    mat("final.norm", d, std=0.2)
    mat("head", cfg["vocab"], d)
    return w


def write_model(directory, cfg, w):
    """config.json + model.safetensors (bf16) of a case."""
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, off = {}, [], 0
    for name, t in w.items():
        b = t.bfloat16().contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    hb = json.dumps(head).encode()
    with open(os.path.join(directory, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(hb)) + hb + b"".join(blobs))
    return str(directory)


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()
