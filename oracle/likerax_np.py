"""Plain NumPy statement of the Likerax decoder, one function per mechanism, float64 throughout.

A model is a dict: ``cfg`` (the config.json dictionary) and ``w`` (tensor name -> array).  Every
function takes whole sequences and loops where a loop says it best; nothing is shared with the
product code.  ``forward`` returns the logits of every position; with ``trace`` it also returns the
residual stream (the sum of the streams) after every layer run.
"""
from __future__ import annotations

import math

import numpy as np


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps), times ``weight`` if there is one; the mean runs over the last axis."""
    x = np.asarray(x, dtype=np.float64)
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def linear(w, x):
    return x @ np.asarray(w, dtype=np.float64).T


def distance_slope(head, heads):
    """Slope of the distance bias of query head ``head`` of ``heads``."""
    return 2.0 ** (-8.0 * (head + 1) / heads)


def visible(i, j, chunk):
    """Whether the query at position i sees the key at position j: not ahead of it, same chunk."""
    return j <= i and (chunk is None or i // chunk == j // chunk)


def attention_head(q, k, v, scale, slope, chunk):
    """One head over one sequence: q [T, D], k [T, D], v [T, V] -> [T, V], one query at a time."""
    out = np.zeros((q.shape[0], v.shape[1]))
    for i in range(q.shape[0]):
        keys = [j for j in range(q.shape[0]) if visible(i, j, chunk)] if chunk else list(range(i + 1))
        s = np.array([float(q[i] @ k[j]) * scale - slope * (i - j) for j in keys])
        p = np.exp(s - s.max())
        out[i] = (p / p.sum()) @ v[keys]
    return out


def attention(w, pre, mixer, eps, h):
    """The whole mixer on h [T, width]."""
    heads, groups, dim, vdim = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    t = h.shape[0]
    mask = mixer.get("mask") or {}
    q = rms_norm(linear(w[pre + "q"], h).reshape(t, heads, dim), None, eps)
    k = rms_norm(linear(w[pre + "k"], h).reshape(t, groups, dim), None, eps)
    v = linear(w[pre + "v"], h).reshape(t, groups, vdim)
    out = np.zeros((t, heads, vdim))
    for a in range(heads):
        g = a // (heads // groups)
        out[:, a] = attention_head(q[:, a], k[:, g], v[:, g], mixer["scale"], distance_slope(a, heads),
                                   mask.get("size"))
    return linear(w[pre + "o"], out.reshape(t, heads * vdim))


def feed_forward(w, pre, h):
    return linear(w[pre + "down"], gelu_tanh(linear(w[pre + "gate"], h)) * linear(w[pre + "up"], h))


def hyper_connection(streams, w_in, w_mix, w_out, sublayer):
    """streams: list of [T, width].  The sublayer reads a weighted sum of the streams; every new stream
    is a mix of all old ones (``w_mix`` is indexed [from][to]) plus its share of the sublayer's output."""
    n = len(streams)
    u = sum(w_in[s] * streams[s] for s in range(n))
    y = sublayer(u)
    return [sum(w_mix[s][t] * streams[s] for s in range(n)) + w_out[t] * y for t in range(n)]


def layer_order(cfg):
    """Layer indices in the order they run: the looped range repeats in place."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


def run_layer(w, cfg, index, streams):
    entry, pre, eps = cfg["layers"][index], f"l{index}.", cfg["norm"]["eps"]

    def hc(q, sub):
        return hyper_connection(streams, w[f"{pre}hc{q}.in"], w[f"{pre}hc{q}.mix"], w[f"{pre}hc{q}.out"],
                                lambda u: sub(rms_norm(u, w[f"{pre}norm{q}"], eps)))

    streams = hc(1, lambda x: attention(w, pre + "mix.", entry["mixer"], eps, x))
    if entry.get("mlp"):
        streams = hc(2, lambda x: feed_forward(w, pre + "mlp.", x))
    return streams


def forward(model, tokens, trace=False):
    """Logits [T, vocab] of one sequence."""
    cfg = model["cfg"]
    w = {n: np.asarray(a, dtype=np.float64) for n, a in model["w"].items()}
    x = w["embed"][np.asarray(tokens, dtype=np.int64)]
    streams = [x.copy() for _ in range(cfg["streams"])]
    seen = []
    for index in layer_order(cfg):
        streams = run_layer(w, cfg, index, streams)
        seen.append(sum(streams))
    logits = linear(w["head"], rms_norm(sum(streams), w["final.norm"], cfg["norm"]["eps"]))
    return (logits, np.stack(seen)) if trace else logits


def generate_greedy(model, prompt, n):
    """n tokens, each the lowest index among the largest logits of the last position, from scratch."""
    seq = [int(t) for t in prompt]
    for _ in range(n):
        seq.append(int(np.argmax(forward(model, seq)[-1])))
    return seq[len(prompt):]
