"""Seeded Miborax models for the tests: a configuration, bf16-representable weights, and a writer of the
config.json + model.safetensors pair the loader reads.

The experts a token gets never rest on a close call: a few columns of the embedding, which no layer writes to,
hold a permutation of well separated values per token, and the routers read those."""
import json
import os

import numpy as np

from likerax_models import bf16


def experts(n=5, top=2, ff=48):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}}


def full(heads=3, dim=24, rot=8, vdim=40, rank=48, q_rank=36, base=9000.0, scale=0.4, mlp="default"):
    """A layer over the whole past: query latent, output gate."""
    return {"type": "latent_attention", "mlp": experts() if mlp == "default" else mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot}}}


def window(size, heads=5, dim=16, rot=12, vdim=24, rank=40, base=700.0, scale=0.5, kv_from=None, mlp="default"):
    e = {"type": "latent_attention_2", "mlp": experts() if mlp == "default" else mlp,
         "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "mask": {"size": size},
                   "rot": {"base": base, "dims": rot}}}
    if kv_from is not None:
        e["mixer"]["kv_from"] = kv_from
    return e


def config(layers, vocab=139, width=88, eps=1e-4, scale=3.0):
    return {"architecture": "Miborax", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": layers}


def make(cfg, seed=0):
    """{cfg, w}: scores of several units, sinks that weigh about as much as a few keys, sublayers that move the
    residual by a few tenths of its size."""
    g = np.random.default_rng(seed)
    d, n = cfg["width"], cfg["vocab"]
    coded = max([e["mlp"]["router"]["experts"] for e in cfg["layers"] if e["mlp"]] + [0])
    assert coded < d
    size = 1 / cfg["embedding"]["scale"]
    embed = size * g.standard_normal((n, d))
    values = np.linspace(-1.5, 1.5, coded) if coded > 1 else np.zeros(coded)
    for t in range(n):
        embed[t, :coded] = size * values[g.permutation(coded)]
    w = {"embed": embed}

    def mat(out, inn, gain=1.0):
        return gain * g.standard_normal((out, inn)) / np.sqrt(inn)

    def closed(m):   # the coded columns keep what the embedding put there
        m[:coded] = 0
        return m

    def norm(name):
        w[name], w[name + ".b"] = 1 + 0.2 * g.standard_normal(d), 0.3 * g.standard_normal(d)
        w[name][:coded], w[name + ".b"][:coded] = 1, 0

    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}."
        x, rows = p + "mix.", m["heads"] * (m["dim"] + m["rot_dim"])
        norm(p + "norm1")
        norm(p + "norm2")
        if "q_rank" in m:
            w[x + "dq"], w[x + "dq.norm"] = mat(m["q_rank"], d), 1 + 0.2 * g.standard_normal(m["q_rank"])
            w[x + "uq"] = mat(rows, m["q_rank"])
            w[x + "g"] = mat(m["heads"], d)
        else:
            w[x + "q"] = mat(rows, d)
        if m.get("kv_from") is None:
            w[x + "dkv"], w[x + "dkv.norm"] = mat(m["kv_rank"] + m["rot_dim"], d), 1 + 0.2 * g.standard_normal(m["kv_rank"])
        w[x + "uk"], w[x + "uv"] = mat(m["heads"] * m["dim"], m["kv_rank"]), mat(m["heads"] * m["vdim"], m["kv_rank"])
        w[x + "sink"] = 1 + g.standard_normal(m["heads"])
        w[x + "o"] = closed(mat(d, m["heads"] * m["vdim"], 0.7))
        if e["mlp"]:
            k, ff = e["mlp"]["router"]["experts"], e["mlp"]["expert"]["ff"]
            for q in range(k):
                w[f"{p}mlp.e{q}.gate"], w[f"{p}mlp.e{q}.up"] = mat(ff, d, 1.5), mat(ff, d)
                w[f"{p}mlp.e{q}.down"] = closed(mat(d, ff))
            w[p + "mlp.router"] = np.eye(k, d)
            w[p + "mlp.router.b"] = 0.02 * g.standard_normal(k)
    norm("final.norm")
    return {"cfg": cfg, "w": {k: bf16(a) for k, a in w.items()}}


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
    from rotor_b200.miborax import MiboraxConfig, build
    return build(MiboraxConfig.from_dict(model["cfg"]), lambda n: torch.from_numpy(model["w"][n]), **kw)
