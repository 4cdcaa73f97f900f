"""The Miborax design: config.json reader and weight loading into a ``DecoderModel``.

Miborax is a decoder whose attention and feed-forward read the same residual, each through a layer norm of its
own.  Attention is latent (a position's cache row is one normed latent and one rotated key part for all heads)
with a sink per head: over the whole past, with queries through a latent and a gate on every head's output
(``latent_attention``), or over a window (``latent_attention_2``), where a layer may read the rows another layer
cached.  The feed-forward is a mixture of experts; the head is the embedding table.
"""
from __future__ import annotations

from dataclasses import dataclass
from pathlib import Path
from typing import List, Optional

from .decoder_model import DecoderModel, Experts, Latent, LayerSpec

MIXERS = ("latent_attention", "latent_attention_2")


@dataclass
class MiboraxExperts:
    experts: int
    top: int
    ff: int


@dataclass
class MiboraxLayer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: Optional[int]     # latent of the queries (the kind over the whole past)
    base: float
    scale: float
    window: int               # 0: every position up to its own
    gated: bool
    kv_from: Optional[int]    # layer whose cache is read
    mlp: Optional[MiboraxExperts]


@dataclass
class MiboraxConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: List[MiboraxLayer]

    @classmethod
    def from_dict(cls, c):
        return cls(c["vocab"], c["width"], float(c["norm"]["eps"]), float((c.get("embedding") or {}).get("scale", 1.0)),
                   [cls._layer(i, e) for i, e in enumerate(c["layers"])])

    @staticmethod
    def _layer(i, e):
        if e["type"] not in MIXERS:
            raise ValueError(f"layer {i}: mixer {e['type']!r} is not part of this design")
        m, mlp, experts = e["mixer"], e.get("mlp"), None
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError(f"layer {i}: {m['rot']['dims']} of {m['rot_dim']} rotated columns turn; this design turns them all")
        if mlp is not None:
            if mlp.get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: feed-forward {mlp['kind']!r} is not part of this design")
            experts = MiboraxExperts(mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"])
        full = e["type"] == "latent_attention"
        return MiboraxLayer(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"] if full else None,
                            float(m["rot"]["base"]), float(m["scale"]), 0 if full else int(m["mask"]["size"]), full,
                            m.get("kv_from"), experts)


def build(cfg: MiboraxConfig, get, **kw) -> DecoderModel:
    """Model from a configuration and ``get(tensor name) -> torch tensor``."""
    layers = []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        x = p + "mix."
        a = Latent(l.kv_rank, l.rot_dim, l.base, get(x + "uk"), get(x + "uv"), kv_from=l.kv_from)
        if l.kv_from is None:
            a.dkv, a.kv_norm = get(x + "dkv"), get(x + "dkv.norm")
        if l.q_rank is not None:
            a.dq, a.q_norm, a.uq = get(x + "dq"), get(x + "dq.norm"), get(x + "uq")
            if a.dq.shape[0] != l.q_rank:
                raise ValueError(f"layer {i}: query latent of {a.dq.shape[0]}, the configuration says {l.q_rank}")
        if l.gated:
            a.gate = get(x + "g")
        spec = LayerSpec(l.heads, 1, l.dim, l.vdim, l.scale, get(x + "q") if l.q_rank is None else None, None, None, get(x + "o"),
                         get(p + "norm1"), window=l.window, sinks=get(x + "sink"), norm1_b=get(p + "norm1.b"), parallel=True, latent=a,
                         act="silu")
        if l.mlp is not None:
            f = p + "mlp."
            each = lambda name: [get(f"{f}e{e}.{name}") for e in range(l.mlp.experts)]
            spec.experts = Experts(l.mlp.top, get(f + "router"), each("gate"), each("up"), each("down"), bias=get(f + "router.b"))
            if spec.experts.gate[0].shape[0] != l.mlp.ff:
                raise ValueError(f"layer {i}: experts of {spec.experts.gate[0].shape[0]} channels, the configuration says {l.mlp.ff}")
            spec.norm2, spec.norm2_b = get(p + "norm2"), get(p + "norm2.b")
        layers.append(spec)
    embed = get("embed")
    if tuple(embed.shape) != (cfg.vocab, cfg.width):
        raise ValueError(f"embedding of shape {tuple(embed.shape)}, the configuration says {(cfg.vocab, cfg.width)}")
    return DecoderModel(layers, range(len(layers)), embed, None, get("final.norm"), eps=cfg.eps, embed_scale=cfg.embed_scale,
                        final_norm_b=get("final.norm.b"), **kw)


def load_miborax_model(model_dir, config, *, dtype="bfloat16", **kw) -> DecoderModel:
    from safetensors import safe_open
    with safe_open(str(Path(model_dir) / "model.safetensors"), framework="pt") as f:
        return build(MiboraxConfig.from_dict(config), f.get_tensor, dtype=dtype, **kw)
