"""GPU: Miborax through the framework against the plain oracle (oracle/miborax_np.py)."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import miborax_models as M
from likerax_models import bf16
from oracle import miborax_np as O
from test_gpu_likerax import Attn, dev, feed, ld, rel, tol

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL, BF16_TOL = 2e-5, 3e-2     # of the RMS; every sublayer's rounding included


# ------------------------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("n,rows", [(64, 3), (100, 5), (1536, 2), (320, 700), (90, 1)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_residual_two_layer_norms(n, rows, dtype):
    """x + y + y2 and both normed rows; then the same from the scaled embedding."""
    import torch
    from rotor_b200 import abi
    g = np.random.default_rng(n + rows)
    x, y, y2 = (g.standard_normal((rows, n)).astype(np.float32) + 2 for _ in range(3))
    w1, b1, w2, b2 = (g.standard_normal(n).astype(np.float32) for _ in range(4))
    table, ids = bf16(g.standard_normal((29, n))), g.integers(0, 29, rows)
    pad = lambda a: dev(a, cols=ld(n))
    xd, yd, y2d, w1d, b1d, w2d, b2d = map(pad, (x, y, y2, w1, b1, w2, b2))
    td, idd = dev(table, "bfloat16", ld(n)), dev(ids.astype(np.int64))
    t, eps = getattr(torch, dtype), 1e-2
    for source in (x + y + y2, 3.7 * table[ids].astype(np.float64)):
        first = source.dtype == np.float64
        xo = torch.zeros((rows, ld(n)), device="cuda")
        h, h2 = (torch.full((rows, ld(n)), float("nan"), dtype=t, device="cuda") for _ in range(2))
        abi.check(abi.lib.rotor_b200_norm_stage(abi.ptr(idd) if first else None, abi.ptr(td), 29, 3.7, abi.ptr(xd), abi.ptr(xo), abi.ptr(yd),
                                                abi.ptr(y2d), abi.ptr(w1d), abi.ptr(b1d), abi.ptr(w2d), abi.ptr(b2d), eps, rows, n, abi.ptr(h),
                                                abi.ptr(h2), int(dtype == "float32"), abi.stream()))
        assert rel(xo.cpu().numpy()[:, :n], source) < 1e-6
        for out, w, b in ((h, w1, b1), (h2, w2, b2)):
            out = out.float().cpu().numpy()
            assert rel(out[:, :n], O.layer_norm(source, w, b, eps)) < (2e-6 if dtype == "float32" else 4e-3)
            assert not out[:, n:].any()


class Mixer:
    """The latent mixer of one layer through the C entry point; the model supplies the packed layer and its cache."""

    def __init__(self, entry, w, dtype, width=88, batch=1, max_seq=256, eps=1e-4):
        import torch
        from rotor_b200 import abi
        self.entry, self.eps, self.dtype, self.width, self.batch, self.max_seq = entry, eps, dtype, width, batch, max_seq
        self.m = M.make(M.config([dict(entry, mlp=None)], width=width, vocab=8, eps=eps), seed=4)
        self.m["w"].update({"l0.mix." + k: bf16(a) for k, a in w.items()})
        self.model = M.load(self.m, dtype=dtype, max_seq=max_seq, max_batch=batch, max_rows=batch * max_seq)
        self.h = self.model._ensure_handle(batch, max_seq, max_seq)
        self.layer = self.model._layers[0]
        need = abi.lib.rotor_b200_decoder_layer_workspace_bytes(C.byref(self.h.cfg), C.byref(self.layer))
        assert need
        self.ws = torch.zeros(need, dtype=torch.uint8, device="cuda")

    def run(self, h, past, expanded=-1):
        """h [batch, seq, width]"""
        import torch
        from rotor_b200 import abi
        b, t = h.shape[:2]
        hd = dev(h.reshape(b * t, -1).astype(np.float32), self.dtype, ld(self.width))
        y = torch.zeros((b * t, ld(self.width)), device="cuda")
        abi.check(abi.lib.rotor_b200_latent_mixer(C.byref(self.h.cfg), C.byref(self.layer), abi.ptr(hd), b, t, past,
                                                  abi.ptr(self.model.runs[0].k_cache), expanded, abi.ptr(y), abi.ptr(self.ws), self.ws.numel(),
                                                  abi.stream()))
        abi.device_status()
        return y.cpu().numpy()[:, :self.width].reshape(b, t, self.width)

    def want(self, h, entry=None):
        """Oracle over one whole sequence [T, width]."""
        w, mixer = self.m["w"], (entry or self.entry)["mixer"]
        h = h.astype(np.float64)
        return O.latent_attention(w, "l0.mix.", mixer, self.eps, h, O.latent_rows(w, "l0.mix.", mixer, self.eps, h))


MIXERS = {
    "window": lambda: M.window(21),
    "window of one": lambda: M.window(1, heads=2, dim=8, rot=2, vdim=56),
    "full": lambda: M.full(),
    "wide": lambda: M.full(heads=4, dim=128, rot=64, vdim=128, rank=320, q_rank=200, scale=0.1),
    "no multiple of anything": lambda: M.window(33, heads=3, dim=21, rot=10, vdim=13, rank=27),
    "more heads than a tile": lambda: M.full(heads=35, dim=8, rot=4, vdim=8, rank=16, q_rank=17),
    "long latent": lambda: M.window(50, heads=2, dim=40, rot=36, vdim=72, rank=600),
    "heads beyond the prompt kernel": lambda: M.window(40, heads=2, dim=136, rot=16, vdim=24, rank=80),
    "rotated part beyond the prompt kernel": lambda: M.full(heads=2, dim=32, rot=72, vdim=160, rank=64),
}


def random_mixer(entry, seed, width=88):
    """Weights of one mixer of its own, with scores of several units."""
    m = M.make(M.config([dict(entry, mlp=None)], width=width, vocab=8), seed=seed)
    return {k[len("l0.mix."):]: a for k, a in m["w"].items() if k.startswith("l0.mix.")}


def poison(tensor):
    """Rows that the product has not written must not matter: fill them with what would show."""
    tensor.fill_(float("nan"))


@pytest.mark.parametrize("name", list(MIXERS))
@pytest.mark.parametrize("dtype,expanded", [("float32", -1), ("bfloat16", -1), ("bfloat16", 0)])
def test_latent_mixer_prompt_portions_and_single_tokens(name, dtype, expanded):
    entry, t = MIXERS[name](), 171
    g = np.random.default_rng(len(name))
    a = Mixer(entry, random_mixer(entry, 7), dtype, max_seq=192)
    h = bf16(g.standard_normal((t, 88)))
    want = a.want(h)
    for sizes in ((90, 2, 17, 1, 1, 40, 3, 1, 1, 1, 14), (1, 1, 1, 1, 2, 1, 5, 16, 143), (171,)):
        poison(a.model.runs[0].k_cache)
        got, at = [], 0
        for n in sizes:
            got.append(a.run(h[None, at:at + n], at, expanded)[0])
            at += n
        assert at == t
        assert rel(np.concatenate(got), want) < tol(dtype), sizes


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("batch", [2, 4, 7, 18])
def test_latent_mixer_of_a_batch_matches_each_alone(batch, dtype):
    """Prompt, short portion and single tokens of several sequences in one call (few rows and many rows)."""
    entry, t = M.window(19, heads=6, rank=72, vdim=32), 62
    g = np.random.default_rng(batch)
    a = Mixer(entry, random_mixer(entry, 9), dtype, batch=batch, max_seq=80)
    poison(a.model.runs[0].k_cache)
    h = bf16(g.standard_normal((batch, t, 88)))
    got, at = [], 0
    for n in (40, 1, 1, 3, 17):
        got.append(a.run(h[:, at:at + n], at))
        at += n
    got = np.concatenate(got, 1)
    for b in range(batch):
        assert rel(got[b], a.want(h[b])) < tol(dtype) / 2, b


def pointed(entry, width, gain):
    """Mixer weights under which the left half of a row asks and the right half answers: the score of i for j is
    large exactly where i's left half is j's right half.  The rotated part keeps out of it."""
    m, half, g = entry["mixer"], width // 2, np.random.default_rng(3)
    w = random_mixer(entry, 5, width)
    heads, dim, rot, rank = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    basis = g.standard_normal((rank, half)) / np.sqrt(half)
    w["dkv"] = np.concatenate([np.concatenate([np.zeros((rank, half)), basis], 1), 0.1 * w["dkv"][rank:]])
    w["dkv.norm"] = np.ones(rank)
    uk = w["uk"].reshape(heads, dim, rank)
    q = np.zeros((heads, dim + rot, width))
    q[:, :dim, :half] = gain * (uk @ basis) / dim
    if "q_rank" in m:    # through a latent that keeps the left half
        w["dq"], w["dq.norm"] = np.eye(m["q_rank"], width), np.ones(m["q_rank"])
        w["uq"] = q.reshape(-1, width)[:, :m["q_rank"]]
    else:
        w["q"] = q.reshape(-1, width)
    w["sink"] = np.zeros(heads)
    return w


EDGES = [(0, 169), (0, 63), (0, 64), (63, 64), (100, 163), (100, 164), (64, 127), (64, 128), (105, 169), (106, 169), (127, 128), (5, 5)]


@pytest.mark.parametrize("dtype,expanded", [("float32", -1), ("bfloat16", -1), ("bfloat16", 0)])
@pytest.mark.parametrize("kind", ["window", "full"])
def test_one_key_stands_out_inside_and_outside_the_window(kind, dtype, expanded):
    """Key `key` is the only one query `query` asks for: visible, it takes nearly the whole weight; past the window
    none.  As a prompt, behind a prompt as a short portion, and as a decoded token."""
    width, size, t = 128, 64, 170
    entry = M.window(size, heads=3, dim=48, rot=8, vdim=40, rank=64, scale=1.0) if kind == "window" else \
        M.full(heads=3, dim=48, rot=8, vdim=40, rank=64, q_rank=64, scale=1.0)
    w = pointed(entry, width, 16.0)
    a = Mixer(entry, w, dtype, width=width, max_seq=192)
    for key, query in EDGES:
        g = np.random.default_rng(key * 200 + query)
        h = g.standard_normal((t, width))
        h[query, :64] = h[key, 64:]
        h = bf16(h)
        want = a.want(h)
        lo = max(0, query - size + 1) if kind == "window" else 0
        # what the output would be if the key were hidden, to see that the input shows what it is meant to show
        moved = h.copy()
        moved[key, 64:] = bf16(g.standard_normal(64))
        told = rel(want[query:query + 1], a.want(moved)[query:query + 1])
        assert (told > 0.5) == (lo <= key) or key == query, (key, query, told)
        got = a.run(h[None], 0, expanded)[0]
        assert rel(got, want) < tol(dtype), (key, query)
        for n in (1, 2):
            poison(a.model.runs[0].k_cache)
            start = max(query - n + 1, 0)
            if start:
                a.run(h[None, :start], 0, expanded)
            one = a.run(h[None, start:query + 1], start, expanded)[0]
            assert rel(one[-1:], want[query:query + 1]) < tol(dtype), (key, query, n)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sinks_of_every_size(dtype):
    """From none to one that takes everything, heads unlike each other; the first tokens have few other keys."""
    entry = M.window(30, heads=5)
    w = random_mixer(entry, 11)
    w["sink"] = np.array([-90.0, -1.0, 2.0, 6.0, 95.0])
    a = Mixer(entry, w, dtype, max_seq=96)
    h = bf16(np.random.default_rng(0).standard_normal((60, 88)))
    want = a.want(h)
    none = dict(a.m["w"], **{"l0.mix.sink": np.full(5, -90.0)})
    assert rel(want, O.latent_attention(none, "l0.mix.", entry["mixer"], a.eps, h.astype(np.float64),
                                        O.latent_rows(none, "l0.mix.", entry["mixer"], a.eps, h.astype(np.float64)))) > 0.3
    for sizes in ((60,), (1, 1, 1, 2, 55), (20, 40)):
        got, at = [], 0
        for n in sizes:
            got.append(a.run(h[None, at:at + n], at)[0])
            at += n
        assert rel(np.concatenate(got), want) < tol(dtype) / 2, sizes


@pytest.mark.parametrize("dtype,row_kernel", [("float32", 1), ("bfloat16", 0), ("bfloat16", 1)])
@pytest.mark.parametrize("dim,vdim,chunk,window", [(64, 64, 0, 37), (128, 40, 60, 25), (160, 136, 0, 48), (32, 32, 0, 0)])
def test_bias_attention_takes_windows_and_sinks_too(dim, vdim, chunk, window, dtype, row_kernel):
    g = np.random.default_rng(dim + vdim)
    heads, kv, t = 4, 2, 130
    q, k, v = (bf16(g.standard_normal((t, n, d))) for n, d in ((heads, dim), (kv, dim), (kv, vdim)))
    slopes, sinks = [0.05, 0.02, 0.01, 0.0], [-3.0, 1.0, 4.0, 2.0]
    a = Attn(heads, kv, dim, vdim, chunk, 0.3, slopes, dtype, max_seq=160, unit=False)
    sd = dev(np.array(sinks, dtype=np.float32))
    a.c.window, a.c.sinks = window, sd.data_ptr()
    want = np.zeros((t, heads, vdim))
    for i in range(t):
        keys = [j for j in range(i + 1) if (not chunk or j // chunk == i // chunk) and O.visible(i, j, window or None)]
        for h in range(heads):
            s = np.array([q[i, h].astype(np.float64) @ k[j, h // 2] * 0.3 - slopes[h] * (i - j) for j in keys])
            want[i, h] = O.sink_softmax(s, sinks[h]) @ v[keys, h // 2].astype(np.float64)
    got, at = [], 0
    for n in (70, 1, 2, 36, 1, 1, 19):
        got.append(a.run(q[None, at:at + n], k[None, at:at + n], v[None, at:at + n], [at], row_kernel)[0])
        at += n
    assert at == t
    assert rel(np.concatenate(got).reshape(t, -1), want.reshape(t, -1)) < tol(dtype) / 2


@pytest.mark.parametrize("n,top,ff,width", [(5, 2, 48, 88), (1, 1, 40, 64), (7, 1, 200, 130), (6, 6, 24, 96), (40, 8, 72, 136), (150, 32, 16, 232)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_experts(n, top, ff, width, dtype):
    """Routed feed-forward of few rows, many rows, and more rows than one tile per expert; rows given as they are, so
    that the choice rests on exact inputs."""
    import torch
    from rotor_b200 import abi
    g = np.random.default_rng(n * top + ff)
    m = M.make(M.config([M.window(4, mlp=M.experts(n, top, ff))], width=width, vocab=8), seed=1)
    m["w"]["l0.mlp.router"] = bf16(2 * g.standard_normal((n, width)) / np.sqrt(width))
    m["w"]["l0.mlp.router.b"] = bf16(0.5 * g.standard_normal(n))
    rows_max = 700
    model = M.load(m, dtype=dtype, max_seq=rows_max, max_rows=rows_max)
    cfg, layer = model._ensure_handle(1, rows_max, rows_max).cfg, model._layers[0]
    need = abi.lib.rotor_b200_decoder_layer_workspace_bytes(C.byref(cfg), C.byref(layer))
    ws = torch.zeros(need, dtype=torch.uint8, device="cuda")
    w = {k: a.astype(np.float64) for k, a in m["w"].items()}
    for rows in (1, 2, 4, 5, 33, rows_max):
        h = bf16(g.standard_normal((rows, width)))
        hd = dev(h, dtype, ld(width))
        y = torch.zeros((rows, ld(width)), device="cuda")
        for _ in range(2):      # (the counts are left ready for the next call)
            abi.check(abi.lib.rotor_b200_experts(C.byref(cfg), C.byref(layer), abi.ptr(hd), rows, abi.ptr(y), abi.ptr(ws), need, abi.stream()))
        abi.device_status()
        z = np.sort(O.linear(w["l0.mlp.router"], h.astype(np.float64)) + w["l0.mlp.router.b"], -1)
        clear = np.ones(rows, bool) if top == n else z[:, n - top] - z[:, n - top - 1] > 1e-4
        assert clear.mean() > 0.9
        want = O.mixture(w, "l0.mlp.", top, h.astype(np.float64))
        assert rel(y.cpu().numpy()[clear, :width], want[clear]) < (5e-6 if dtype == "float32" else 1.5e-2), rows


# ------------------------------------------------------------------------------- whole models
CONFIGS = {
    "mixed": lambda: M.config([M.window(24), M.window(17, kv_from=0, heads=2, dim=28, vdim=36), M.full(),
                               M.window(24, kv_from=0, mlp=None), M.window(31, mlp=M.experts(7, 3, 40)), M.window(9, kv_from=4, heads=7)]),
    "a full layer lends its cache": lambda: M.config([M.full(heads=2, dim=16, rot=12, rank=40, base=700.0, mlp=M.experts(4, 4, 24)),
                                                      M.window(40, kv_from=0, heads=4), M.window(1)], width=264, vocab=64, scale=1.0),
    "large heads": lambda: M.config([M.full(heads=3, dim=128, rot=64, vdim=128, rank=256, q_rank=96, scale=0.1, mlp=M.experts(3, 1, 136)),
                                     M.window(70, heads=17, dim=64, rot=32, vdim=64, rank=128, scale=0.2, mlp=M.experts(12, 6, 64))],
                                    width=192, vocab=300, eps=1e-3, scale=0.5),
    "one expert": lambda: M.config([M.full(heads=1, dim=8, rot=2, vdim=8, rank=8, q_rank=8, mlp=M.experts(1, 1, 8)),
                                    M.window(1000, heads=1, dim=8, rot=2, vdim=8, rank=8, base=40.0)], width=72, vocab=31),
}


@pytest.fixture(scope="module")
def case():
    cache = {}

    def get(name, dtype):
        if name not in cache:
            m = M.make(CONFIGS[name](), seed=len(name))
            toks = np.random.default_rng(1).integers(0, m["cfg"]["vocab"], 123)
            cache[name] = (m, toks, O.forward(m, toks))
        m, toks, want = cache[name]
        if (name, dtype) not in cache:
            cache[name, dtype] = M.load(m, dtype=dtype, max_seq=160)
        return cache[name, dtype], m, toks, want
    return get


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [[123], [1], [2], [3], [60, 2, 16, 1, 5], [33, 17]], ids=str)
def test_portions_match_the_oracle(case, name, dtype, sizes):
    model, m, toks, want = case(name, dtype)
    assert rel(feed(model, toks, sizes), want) < tol(dtype)


def test_planted_mistakes_would_show(case, monkeypatch):
    """The oracle with one mistake each is far outside the tolerance that the product meets."""
    model, m, toks, want = case("mixed", "bfloat16")
    toks = toks[:70]
    got = feed(model, toks, [70])
    assert rel(got, want[:70]) < BF16_TOL

    def changed(change):
        c, w = json.loads(json.dumps(m["cfg"])), dict(m["w"])
        change(c, w)
        return rel(got, O.forward({"cfg": c, "w": w}, toks))

    def window(c, w):
        c["layers"][0]["mixer"]["mask"]["size"] += 1

    def sink(c, w):
        w["l2.mix.sink"] = np.full(3, -90.0)

    def base(c, w):
        c["layers"][2]["mixer"]["rot"]["base"] /= 3

    def gate(c, w):
        w["l2.mix.g"] = np.zeros_like(w["l2.mix.g"])

    def top(c, w):
        c["layers"][4]["mlp"]["router"]["top"] -= 1

    def router_bias(c, w):
        w["l4.mlp.router.b"] = w["l4.mlp.router.b"] + np.linspace(0, 2, 7)

    def norms(c, w):
        w["l1.norm2"], w["l1.norm2.b"] = w["l1.norm1"], w["l1.norm1.b"]

    def borrowed(c, w):
        c["layers"][5]["mixer"]["kv_from"] = 0

    def scale(c, w):
        c["embedding"]["scale"] *= 1.3

    for change in (window, sink, base, gate, top, router_bias, norms, borrowed, scale):
        assert changed(change) > 2 * BF16_TOL, change.__name__
    with monkeypatch.context() as p:    # one sublayer after the other
        def serial(w, cfg, index, x, caches):
            pre, eps, entry = f"l{index}.", cfg["norm"]["eps"], cfg["layers"][index]
            h = O.layer_norm(x, w[pre + "norm1"], w[pre + "norm1.b"], eps)
            src = entry["mixer"].get("kv_from", index)
            if src == index:
                caches[index] = O.latent_rows(w, pre + "mix.", entry["mixer"], eps, h)
            x = x + O.latent_attention(w, pre + "mix.", entry["mixer"], eps, h, caches[src])
            if entry["mlp"]:
                x = x + O.mixture(w, pre + "mlp.", entry["mlp"]["router"]["top"], O.layer_norm(x, w[pre + "norm2"], w[pre + "norm2.b"], eps))
            return x
        p.setattr(O, "run_layer", serial)
        assert rel(got, O.forward(m, toks)) > 2 * BF16_TOL


def test_a_borrowing_layer_has_no_cache_of_its_own(case):
    model, *_ = case("mixed", "float32")
    model._ensure_handle(1, 1, 1)
    k = [r.k_cache for r in model.runs]
    assert k[1] is k[0] and k[3] is k[0] and k[5] is k[4] and k[2] is not k[0] and k[4] is not k[0]
    assert tuple(k[0].shape) == (1, 1, model.max_seq, 64)     # latent of 40 and rotated 12, each to sixteens


def test_positions_that_are_given_back_are_used_again(case):
    model, m, toks, want = case("mixed", "float32")
    other = np.random.default_rng(9).integers(0, m["cfg"]["vocab"], 140)
    feed(model, other, [140])
    assert rel(feed(model, toks[:40], [11, 1, 2]), want[:40]) < F32_TOL
    feed(model, other, [7])
    assert rel(feed(model, toks, [123]), want) < F32_TOL


def test_the_cache_grows_and_keeps_its_contents(case):
    _, m, toks, want = case("mixed", "float32")
    model = M.load(m, dtype="float32", max_seq=16, max_rows=8)
    assert rel(feed(model, toks, [8, 1, 30]), want) < F32_TOL


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_keys_far_away(dtype):
    """Decoding across many windows behind a prompt longer than one tile of every kernel."""
    m = M.make(M.config([M.full(heads=2), M.window(50, heads=2)], vocab=67), seed=6)
    toks = np.random.default_rng(2).integers(0, 67, 640)
    want = O.forward(m, toks)
    model = M.load(m, dtype=dtype, max_seq=1024)     # (room for the most splits of the attention's cluster)
    assert rel(feed(model, toks, [560] + [1] * 80), want) < tol(dtype)
    assert rel(feed(model, toks[:85], [5] + [1] * 80), want[:85]) < tol(dtype)


def test_api_forward_shapes_and_caches(case):
    model, m, toks, want = case("one expert", "float32")
    both, caches = model.forward(np.stack([toks[:20], toks[20:40]]), use_cache=True)
    assert both.shape == (2, 20, m["cfg"]["vocab"]) and rel(both[0], want[:20]) < F32_TOL
    assert caches[0]["k"].shape == (2, 1, 20, 32)
    with pytest.raises(KeyError):
        caches[0]["v"]
    step, caches = model.forward(np.array([[toks[20]], [toks[40]]]), past_kv_cache=caches, use_cache=True)
    assert rel(step[0], want[20:21]) < F32_TOL and caches[0].length == 21
    assert rel(step[1], O.forward(m, toks[20:41])[-1:]) < F32_TOL


# ------------------------------------------------------------------------------- generation
def greedy_want(m, prompt, n):
    """Oracle generation and the smallest margin between the two best logits on the way."""
    seq, margin = [int(t) for t in prompt], np.inf
    for _ in range(n):
        lg = O.forward(m, seq)[-1]
        top = np.sort(lg)
        margin = min(margin, (top[-1] - top[-2]) / np.sqrt(np.mean(lg ** 2)))
        seq.append(int(np.argmax(lg)))
    return seq[len(prompt):], margin


def test_greedy_generation_through_the_text_generator(case):
    from rotor_b200.generation import TextGenerator, TopKSampling
    from rotor_b200.synth import PassThroughTokenizer
    model, m, toks, _ = case("mixed", "float32")
    prompt, n = toks[:21], 30
    want, margin = greedy_want(m, prompt, n)
    assert margin > 10 * F32_TOL
    for use_cache in (True, False):
        gen = TextGenerator(model, PassThroughTokenizer(), max_length=len(prompt) + n, use_cache=use_cache)
        out = [int(t) for t in gen.generate(" ".join(map(str, prompt)), max_new_tokens=n, stop_on_eos=False).split()]
        assert out[len(prompt):] == want
    assert model.generate_greedy(prompt, n, use_graph=False) == want
    gen = TextGenerator(model, PassThroughTokenizer(), TopKSampling(1, seed=3), max_length=len(prompt) + n)
    out = [int(t) for t in gen.generate(" ".join(map(str, prompt)), max_new_tokens=n, stop_on_eos=False).split()]
    assert out[len(prompt):] == want


@pytest.mark.parametrize("lens", [[3, 21, 24, 48], [1, 30, 17, 2, 64, 25, 23]], ids=["fused step", "seven prompts"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batch_of_unequal_prompts_generates_what_each_does_alone(case, lens, dtype):
    model, m, toks, _ = case("mixed", dtype)
    prompts = [toks[i:i + n] for i, n in enumerate(lens)]
    got = model.generate_greedy_batch(prompts, 12)
    for b, p in enumerate(prompts):
        want, margin = greedy_want(m, p, 12)
        if margin > (10 * F32_TOL if dtype == "float32" else 2 * BF16_TOL):
            assert got[b].tolist() == want, b
        else:
            assert dtype == "bfloat16"      # (a choice too close for 16 bits)
    same = model.generate_greedy_batch([prompts[1]] * 3, 12)
    assert all(r.tolist() == same[0].tolist() for r in same)


def test_unfused_steps_match_the_oracle(case):
    """ROTOR_B200_NO_FUSED_STEP: stages and products as kernels of their own; ROTOR_B200_NO_TCGEN05: prompts absorbed."""
    model, m, toks, want = case("mixed", "bfloat16")
    code = ("import sys, numpy as np, miborax_models as M, test_gpu_miborax as T\n"
            "m = M.make(T.CONFIGS['mixed'](), seed=len('mixed'))\n"
            "toks = np.random.default_rng(1).integers(0, m['cfg']['vocab'], 123)\n"
            "np.save(sys.argv[1], T.feed(M.load(m, max_seq=160), toks, [60, 1, 3]))\n")
    out = os.path.join(os.environ.get("TMPDIR", "/tmp"), f"miborax_unfused_{os.getpid()}.npy")
    path = os.pathsep.join([ROOT, os.path.join(ROOT, "rotor-rag_b200"), os.path.join(ROOT, "tests")])
    try:
        for switch in ("ROTOR_B200_NO_FUSED_STEP", "ROTOR_B200_NO_TCGEN05"):
            subprocess.check_call([sys.executable, "-c", code, out], env=dict(os.environ, PYTHONPATH=path, **{switch: "1"}), cwd=ROOT)
            assert rel(np.load(out), want) < BF16_TOL, switch
    finally:
        if os.path.exists(out):
            os.remove(out)


# ------------------------------------------------------------------------------- files and programs
def test_checkpoint_command_line_and_trace_replay(tmp_path, case, capsys):
    from rotor_b200.__main__ import main
    _, m, toks, want = case("mixed", "float32")
    folder = M.write(m, tmp_path / "model")
    prompt = " ".join(str(int(t)) for t in toks[:21])
    assert main(["generate", "--model", folder, "--dtype", "float32", "--prompt", prompt, "--max-new-tokens", "10"]) == 0
    assert [int(t) for t in capsys.readouterr().out.split()] == greedy_want(m, toks[:21], 10)[0]

    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:70].tolist(), "want": [0, 23, 24, 69]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[70:73].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[73:74].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": toks[:30].tolist(), "want": [29, 1]}], "end": ["b"]}]
    rows = {0: [0, 23, 24, 69], 2: [73], 3: [29, 1]}
    for dtype in ("bfloat16", "float32"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "80"], input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True)
        assert r.returncode == 0, r.stderr
        assert r.stdout.split("\n")[:4] == [f"done {i}" for i in range(4)]
        assert not (out / "1.f32").exists()
        for i, at in rows.items():
            got = np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(len(at), -1)
            assert rel(got, want[at]) < tol(dtype)
