"""Seeded Likerax models for the tests: a configuration, bf16-representable weights, and a writer of the
config.json + model.safetensors pair the loader reads."""
import json
import os

import numpy as np


def bf16(a):
    """Nearest bf16 value of every element, as float32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7fff + ((u >> 16) & 1)) & 0xffff0000
    return u.astype(np.uint32).view(np.float32).reshape(np.shape(a))


def layer(heads=4, kv_heads=2, dim=32, vdim=32, scale=0.3, chunk=24, ff=96):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": chunk}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, vocab=157, width=96, streams=3, eps=1e-5, loop=None):
    c = {"architecture": "Likerax", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "layers": layers}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def make(cfg, seed=0):
    """{cfg, w}: weights scaled so that every sublayer moves the streams by a few tenths of their size."""
    g = np.random.default_rng(seed)
    d, s = cfg["width"], cfg["streams"]
    w = {"embed": g.standard_normal((cfg["vocab"], d)), "head": g.standard_normal((cfg["vocab"], d)) / np.sqrt(d),
         "final.norm": 1 + 0.2 * g.standard_normal(d)}

    def mat(out, inn, gain=1.0):
        return gain * g.standard_normal((out, inn)) / np.sqrt(inn)

    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}."
        w[p + "norm1"] = 1 + 0.2 * g.standard_normal(d)
        w[p + "mix.q"] = mat(m["heads"] * m["dim"], d)
        w[p + "mix.k"] = mat(m["kv_heads"] * m["dim"], d)
        w[p + "mix.v"] = mat(m["kv_heads"] * m["vdim"], d)
        w[p + "mix.o"] = mat(d, m["heads"] * m["vdim"])
        subs = [1]
        if e["mlp"]:
            ff = e["mlp"]["ff"]
            w[p + "norm2"] = 1 + 0.2 * g.standard_normal(d)
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(ff, d, 1.5), mat(ff, d), mat(d, ff)
            subs.append(2)
        for q in subs:
            w[p + f"hc{q}.in"] = 0.5 + 0.4 * g.standard_normal(s)
            w[p + f"hc{q}.out"] = 0.5 + 0.4 * g.standard_normal(s)
            w[p + f"hc{q}.mix"] = 0.9 * np.eye(s) + 0.15 * g.standard_normal((s, s))
    return {"cfg": cfg, "w": {n: bf16(a) for n, a in w.items()}}


def write(model, directory):
    import torch
    from safetensors.torch import save_file
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(model["cfg"], f)
    save_file({n: torch.from_numpy(a).to(torch.bfloat16).contiguous() for n, a in model["w"].items()},
              os.path.join(directory, "model.safetensors"))
    return str(directory)


def load(model, **kw):
    """Straight from the dict, through the product's builder."""
    import torch
    from rotor_b200.likerax import LikeraxConfig, build
    return build(LikeraxConfig.from_dict(model["cfg"]), lambda n: torch.from_numpy(model["w"][n]), **kw)
