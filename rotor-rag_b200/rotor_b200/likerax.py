"""The Likerax design: config.json reader and weight loading into a ``DecoderModel``.

Likerax is a decoder with hyper-connection streams; its attention divides queries and keys by their root
mean square, takes a distance bias of slope 2^(-8 (h + 1) / heads) off the scores and lets a position see
only its own chunk; its feed-forward is gated with the tanh form of gelu; a range of layers can run
several times in a row with the same weights.
"""
from __future__ import annotations

from dataclasses import dataclass
from pathlib import Path
from typing import List, Optional

from .decoder_model import Connections, DecoderModel, LayerSpec


@dataclass
class LikeraxLayer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int
    ff: Optional[int]      # None: the layer has no feed-forward


@dataclass
class LikeraxConfig:
    vocab: int
    width: int
    streams: int
    eps: float
    layers: List[LikeraxLayer]
    order: List[int]       # layer of every run

    @classmethod
    def from_dict(cls, c):
        layers = []
        for i, e in enumerate(c["layers"]):
            if e["type"] != "attention":
                raise ValueError(f"layer {i}: mixer {e['type']!r} is not part of this design")
            m, mlp = e["mixer"], e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: feed-forward {mlp['kind']!r} is not part of this design")
            layers.append(LikeraxLayer(m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]),
                                       int((m.get("mask") or {}).get("size") or 0), None if mlp is None else mlp["ff"]))
        return cls(c["vocab"], c["width"], c.get("streams", 1), float(c["norm"]["eps"]), layers,
                   run_order(len(layers), c.get("loop")))


def run_order(n_layers, loop=None):
    """Layers in the order they run; ``loop`` = {start, stop, times} repeats start .. stop - 1 in place."""
    order = list(range(n_layers))
    if not loop:
        return order
    a, b, times = loop["start"], loop["stop"], loop["times"]
    if not (0 <= a <= b <= n_layers and times >= 0):
        raise ValueError(f"loop {loop} does not fit {n_layers} layers")
    return order[:a] + order[a:b] * times + order[b:]


def distance_slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def build(cfg: LikeraxConfig, get, **kw) -> DecoderModel:
    """Model from a configuration and ``get(tensor name) -> torch tensor``."""
    def hc(pre):
        return Connections(get(pre + "in"), get(pre + "out"), get(pre + "mix"))

    layers = []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        spec = LayerSpec(l.heads, l.kv_heads, l.dim, l.vdim, l.scale, get(p + "mix.q"), get(p + "mix.k"), get(p + "mix.v"),
                         get(p + "mix.o"), get(p + "norm1"), unit_qk=True, chunk=l.chunk, slopes=distance_slopes(l.heads),
                         hc1=hc(p + "hc1."))
        if l.ff is not None:
            spec.gate, spec.up, spec.down = get(p + "mlp.gate"), get(p + "mlp.up"), get(p + "mlp.down")
            if spec.gate.shape[0] != l.ff:
                raise ValueError(f"layer {i}: feed-forward of {spec.gate.shape[0]} channels, the configuration says {l.ff}")
            spec.norm2, spec.hc2 = get(p + "norm2"), hc(p + "hc2.")
        layers.append(spec)
    embed = get("embed")
    if tuple(embed.shape) != (cfg.vocab, cfg.width):
        raise ValueError(f"embedding of shape {tuple(embed.shape)}, the configuration says {(cfg.vocab, cfg.width)}")
    return DecoderModel(layers, cfg.order, embed, get("head"), get("final.norm"), streams=cfg.streams, eps=cfg.eps, **kw)


def load_likerax_model(model_dir, config, *, dtype="bfloat16", **kw) -> DecoderModel:
    from safetensors import safe_open
    with safe_open(str(Path(model_dir) / "model.safetensors"), framework="pt") as f:
        return build(LikeraxConfig.from_dict(config), f.get_tensor, dtype=dtype, **kw)
