"""Plain NumPy statement of the Miborax decoder, one function per mechanism, float64 throughout.

A model is a dict: ``cfg`` (the config.json dictionary) and ``w`` (tensor name -> array).  Every
function takes whole sequences and loops where a loop says it best; nothing is shared with the
product code.  ``forward`` returns the logits of every position; with ``trace`` it also returns the
residual stream after every layer.
"""
from __future__ import annotations

import numpy as np


def layer_norm(x, weight, bias, eps):
    x = np.asarray(x, dtype=np.float64)
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * weight + bias


def rms_norm(x, weight, eps):
    x = np.asarray(x, dtype=np.float64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def linear(w, x):
    return x @ np.asarray(w, dtype=np.float64).T


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rotate(x, positions, base, dims):
    """x [T, ..., D]: the pairs (2i, 2i + 1) below `dims` turn by position * base^(-2i / dims)."""
    out = np.array(x, dtype=np.float64)
    for t, p in enumerate(positions):
        for i in range(dims // 2):
            a = p * float(base) ** (-2.0 * i / dims)
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = u * np.cos(a) - v * np.sin(a)
            out[t, ..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def visible(i, j, window):
    """The query at position i sees the key at j: not ahead of it, and among its last `window` positions."""
    return j <= i and (window is None or i - j < window)


def sink_softmax(scores, sink):
    """Weights of the scores when exp(sink) joins the denominator (None: it does not)."""
    top = scores.max() if sink is None else max(scores.max(), float(sink))
    e = np.exp(scores - top)
    return e / (e.sum() + (0.0 if sink is None else np.exp(float(sink) - top)))


def attention_head(q, k, v, scale, sink, window):
    """One head over one sequence: q, k [T, D], v [T, V] -> [T, V], one query at a time."""
    out = np.zeros((q.shape[0], v.shape[1]))
    for i in range(q.shape[0]):
        lo = next(j for j in range(i + 1) if visible(i, j, window)) if window else 0
        out[i] = sink_softmax(k[lo:i + 1] @ q[i] * scale, sink) @ v[lo:i + 1]
    return out


def latent_rows(w, pre, mixer, eps, h):
    """What a latent cache holds of h [T, width]: normed latents [T, rank] and the turned key part [T, rot_dim]."""
    rank = mixer["kv_rank"]
    z = linear(w[pre + "dkv"], h)
    c = rms_norm(z[:, :rank], w[pre + "dkv.norm"], eps)
    return c, rotate(z[:, rank:], range(len(h)), mixer["rot"]["base"], mixer["rot"]["dims"])


def latent_queries(w, pre, mixer, eps, h):
    """[T, heads, dim + rot_dim], the last part of each head turned; through a latent of its own if there is one."""
    if pre + "dq" in w:
        q = linear(w[pre + "uq"], rms_norm(linear(w[pre + "dq"], h), w[pre + "dq.norm"], eps))
    else:
        q = linear(w[pre + "q"], h)
    dim = mixer["dim"]
    q = q.reshape(len(h), mixer["heads"], dim + mixer["rot_dim"])
    turned = rotate(q[..., dim:], range(len(h)), mixer["rot"]["base"], mixer["rot"]["dims"])
    return np.concatenate([q[..., :dim], turned], axis=-1)


def latent_attention(w, pre, mixer, eps, h, cache):
    """The mixer on h [T, width]; `cache`: the (latents, key part) it reads, its own or another layer's."""
    c, kr = cache
    t, heads, dim, vdim = len(h), mixer["heads"], mixer["dim"], mixer["vdim"]
    q = latent_queries(w, pre, mixer, eps, h)
    k = linear(w[pre + "uk"], c).reshape(t, heads, dim)
    v = linear(w[pre + "uv"], c).reshape(t, heads, vdim)
    window = (mixer.get("mask") or {}).get("size")
    out = np.zeros((t, heads, vdim))
    for a in range(heads):
        key = np.concatenate([k[:, a], kr], axis=-1)
        out[:, a] = attention_head(q[:, a], key, v[:, a], mixer["scale"], w[pre + "sink"][a], window)
    if pre + "g" in w:
        out = out * sigmoid(linear(w[pre + "g"], h))[:, :, None]
    return linear(w[pre + "o"], out.reshape(t, heads * vdim))


def routes(logits, top):
    """[(expert, weight)] of one token: the `top` largest logits (the lower index first among equals), softmax
    over those alone."""
    order = sorted(range(len(logits)), key=lambda e: (-logits[e], e))[:top]
    z = np.array([logits[e] for e in order])
    p = np.exp(z - z.max())
    return list(zip(order, p / p.sum()))


def expert(w, pre, x):
    return linear(w[pre + "down"], silu(linear(w[pre + "gate"], x)) * linear(w[pre + "up"], x))


def mixture(w, pre, top, h):
    out = np.zeros_like(h)
    logits = linear(w[pre + "router"], h) + w[pre + "router.b"]
    for t in range(len(h)):
        for e, p in routes(logits[t], top):
            out[t] += p * expert(w, f"{pre}e{e}.", h[t])
    return out


def run_layer(w, cfg, index, x, caches):
    """Both sublayers read the same x; `caches` holds the latent rows of the layers that make their own."""
    entry, pre, eps = cfg["layers"][index], f"l{index}.", cfg["norm"]["eps"]
    mixer = entry["mixer"]
    h = layer_norm(x, w[pre + "norm1"], w[pre + "norm1.b"], eps)
    source = mixer.get("kv_from")
    if source is None:
        source = index
        caches[index] = latent_rows(w, pre + "mix.", mixer, eps, h)
    y = latent_attention(w, pre + "mix.", mixer, eps, h, caches[source])
    if entry.get("mlp"):
        y = y + mixture(w, pre + "mlp.", entry["mlp"]["router"]["top"],
                        layer_norm(x, w[pre + "norm2"], w[pre + "norm2.b"], eps))
    return x + y


def forward(model, tokens, trace=False):
    """Logits [T, vocab] of one sequence."""
    cfg = model["cfg"]
    w = {n: np.asarray(a, dtype=np.float64) for n, a in model["w"].items()}
    x = w["embed"][np.asarray(tokens, dtype=np.int64)] * cfg["embedding"]["scale"]
    seen, caches = [], {}
    for index in range(len(cfg["layers"])):
        x = run_layer(w, cfg, index, x, caches)
        seen.append(x)
    logits = linear(w["embed"], layer_norm(x, w["final.norm"], w["final.norm.b"], cfg["norm"]["eps"]))
    return (logits, np.stack(seen)) if trace else logits


def generate_greedy(model, prompt, n):
    """n tokens, each the lowest index among the largest logits of the last position, from scratch."""
    seq = [int(t) for t in prompt]
    for _ in range(n):
        seq.append(int(np.argmax(forward(model, seq)[-1])))
    return seq[len(prompt):]
