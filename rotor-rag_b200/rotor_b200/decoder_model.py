"""Decoders described layer by layer, behind one C handle (rotor_b200_decoder_*).

A design is a list of ``LayerSpec`` (sizes, constants and weights of one layer), the order its layers run
in (a layer may run several times, every run with its own cache), and the embedding, head and final norm.
``DecoderModel`` packs the weights for the kernels, owns the caches and shares the forward and generation
API of every other model (``HandleModel``).
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional, Sequence

from . import abi
from .abi import RotorB200Error, check, lib, ptr
from .handle_model import HandleModel
from .transformer import KVCache

DTYPES = ("bfloat16", "float32")


def _round(n, m):
    return (n + m - 1) // m * m


def pack_matrix(parts, columns_to=64):
    """Row-stacked bf16 device matrix; the row stride is the column count rounded up, pads are zero."""
    torch = abi.require_cuda()
    rows, cols = sum(p.shape[0] for p in parts), parts[0].shape[1]
    out = torch.zeros((rows, _round(cols, columns_to)), dtype=torch.bfloat16, device="cuda")
    r = 0
    for p in parts:
        if p.dim() != 2 or p.shape[1] != cols:
            raise ValueError(f"matrix of shape {tuple(p.shape)} where {cols} columns are expected")
        out[r:r + p.shape[0], :cols] = p.to("cuda", torch.bfloat16)
        r += p.shape[0]
    return out


def pack_vector(v, to=1):
    torch = abi.require_cuda()
    v = v.reshape(-1)
    out = torch.zeros(_round(v.numel(), to), dtype=torch.float32, device="cuda")
    out[:v.numel()] = v.to("cuda", torch.float32)
    return out


def pad_rows(t, rows):
    """The matrix with rows of zeros behind it."""
    out = t.new_zeros((rows, t.shape[1]))
    out[:t.shape[0]] = t
    return out


def expect(name, t, shape):
    if tuple(t.shape) != tuple(shape):
        raise ValueError(f"{name} matrix of shape {tuple(t.shape)}, expected {tuple(shape)}")


def rotary_table(positions, rot_dim, base):
    """cos and sin of position * base^(-2i / rot_dim), [positions, rot_dim / 2, 2] on the device (angles in float64)."""
    torch = abi.require_cuda()
    i = torch.arange(rot_dim // 2, dtype=torch.float64)
    a = torch.arange(positions, dtype=torch.float64)[:, None] * (float(base) ** (-2.0 * i / max(rot_dim, 1)))[None]
    return torch.stack([a.cos(), a.sin()], -1).to(torch.float32).cuda().contiguous()


def plan_runs(specs, order):
    """The runs of the layers in ``order``; one whose layer reads another's cache is tied to that layer's last run
    before it."""
    runs, last = [], {}
    for i in map(int, order):
        if not 0 <= i < len(specs):
            raise ValueError(f"run of layer {i}, but there are {len(specs)} layers")
        a, source = specs[i].latent, None
        if a is not None and a.dkv is None:
            if a.kv_from not in last:
                raise ValueError(f"layer {i} reads the cache of layer {a.kv_from}, which does not run before it")
            source = last[a.kv_from]
            b = specs[a.kv_from].latent
            if b is None or b.dkv is None or (b.rank, b.rot_dim, b.base) != (a.rank, a.rot_dim, a.base):
                raise ValueError(f"layer {i} cannot read the cache of layer {a.kv_from}: it holds other rows")
        runs.append(_Run(i, source))
        last[i] = runs[-1]
    return runs


ACTIVATIONS = {"gelu_tanh": abi.ACT_GELU_TANH, "silu": abi.ACT_SILU}


@dataclass
class Connections:
    """Hyper-connection of one sublayer: ``in_`` [streams], ``out`` [streams], ``mix`` [from, to].  None in a
    LayerSpec is the ordinary residual (one stream)."""
    in_: object
    out: object
    mix: object


@dataclass
class Latent:
    """Latent attention of a layer.  ``dkv`` [rank + rot_dim, width] with ``kv_norm`` [rank]: the cached latent
    and rotated key part, or None where ``kv_from`` names the layer whose cache this one reads; ``uk`` [heads dim,
    rank], ``uv`` [heads vdim, rank].  Queries [heads (dim + rot_dim)]: ``q`` of the LayerSpec, or ``uq`` of the
    normed ``dq``.  ``gate`` [heads, width]: sigmoid gate of a head's output, or None.  ``base``: of the rotary
    frequencies base^(-2i / rot_dim), pairs (2i, 2i + 1)."""
    rank: int
    rot_dim: int
    base: float
    uk: object
    uv: object
    dkv: object = None
    kv_norm: object = None
    dq: object = None
    q_norm: object = None
    uq: object = None
    gate: object = None
    kv_from: Optional[int] = None


@dataclass
class Experts:
    """Routed feed-forward: ``gate``, ``up``, ``down`` are lists of the experts' matrices, ``top`` of them serve a
    token by the largest ``router`` h + ``bias``, weighted by the softmax over those."""
    top: int
    router: object
    gate: Sequence
    up: Sequence
    down: Sequence
    bias: object = None


@dataclass
class LayerSpec:
    """One layer.  Matrices are [out, in] torch tensors.  ``slopes``: distance-bias slope per query head, or
    None; ``chunk`` / ``window``: chunk length / window of the mask, or 0; ``sinks``: per head, exp(sink) joins the
    softmax's denominator; ``latent``: latent attention (k, v and slopes are None then); ``gate`` None and
    ``experts`` None: no feed-forward; ``norm1_b`` / ``norm2_b``: layer norms instead of root mean square ones;
    ``parallel``: both sublayers read the same residual."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q: object
    k: object
    v: object
    o: object
    norm1: object
    unit_qk: bool = False
    chunk: int = 0
    slopes: Optional[Sequence[float]] = None
    gate: object = None
    up: object = None
    down: object = None
    norm2: object = None
    hc1: Optional[Connections] = None
    hc2: Optional[Connections] = None
    window: int = 0
    sinks: object = None
    act: str = "gelu_tanh"
    norm1_b: object = None
    norm2_b: object = None
    parallel: bool = False
    latent: Optional[Latent] = None
    experts: Optional[Experts] = None


class _Run:
    """One run of a layer: owner of its caches, unless it reads those of the run ``source``."""

    def __init__(self, layer, source=None):
        self.layer, self.source = layer, source
        self.k_cache = self.v_cache = None


class _DecoderHandle:
    """Owns one decoder handle and the device workspace it points into."""

    def __init__(self, model, max_batch, max_seq, max_rows):
        torch = abi.require_cuda()
        for run in model.runs:
            model._grow_cache(run, max_batch, max_seq)
        self.cfg = abi.DecoderConfig(vocab_size=model.vocab_size, width=model.width, streams=model.streams,
                                     n_layers=len(model._layers), n_runs=len(model.runs),
                                     f32=int(model.dtype == "float32"), eps=model.eps, max_batch=max_batch,
                                     max_seq=max_seq, max_rows=max_rows, embed_scale=model.embed_scale,
                                     final_norm_b=ptr(model._final_norm_b))
        rope = {}             # one table per (rotary size, base) of the layers
        for s, c in zip(model.specs, model._layers):
            if s.latent is not None:
                key = (s.latent.rot_dim, s.latent.base)
                if key not in rope:
                    rope[key] = rotary_table(max_seq, *key)
                c.rope = ptr(rope[key])
        layers = (abi.DecoderLayer * len(model._layers))(*model._layers)
        runs = (abi.DecoderRun * len(model.runs))()
        for r, run in zip(runs, model.runs):
            r.layer, r.k_cache, r.v_cache = run.layer, ptr(run.k_cache), ptr(run.v_cache)
        need = lib.rotor_b200_decoder_workspace_bytes(C.byref(self.cfg), layers)
        if need == 0:
            raise RotorB200Error("decoder shape not supported by the GPU path (width up to 10240, up to 16 streams, "
                                 "head sizes up to 512, latents up to 1024, up to 1024 experts and 32 per token)")
        self.workspace = torch.empty(need, dtype=torch.uint8, device="cuda")
        self.keep = (model._tensors, rope, [(r.k_cache, r.v_cache) for r in model.runs])  # the handle points into these
        h = C.c_void_p()
        check(lib.rotor_b200_decoder_create(C.byref(self.cfg), layers, runs, ptr(model._embed), ptr(model._head),
                                            ptr(model._final_norm), ptr(self.workspace), need, C.byref(h)),
              "decoder_create")
        self.h = h

    def __del__(self):
        h, self.h = getattr(self, "h", None), None
        if h and lib is not None:   # (module globals are gone at interpreter exit)
            lib.rotor_b200_model_destroy(h)


class DecoderModel(HandleModel):
    """``order``: layer index of every run, in the order they run.  ``head`` None: the embedding table, which the
    input takes times ``embed_scale``."""

    def __init__(self, layers: Sequence[LayerSpec], order: Sequence[int], embed, head, final_norm, *, streams: int = 1,
                 eps: float = 1e-6, embed_scale: float = 1.0, final_norm_b=None, dtype: str = "bfloat16", max_seq: int = 2048, max_batch: int = 1,
                 max_rows: Optional[int] = None):
        torch = abi.require_cuda()
        if dtype not in DTYPES:
            raise ValueError(f"dtype {dtype!r} is not one of {DTYPES}")
        if not layers or not order:
            raise ValueError("a decoder needs at least one layer and one run")
        self.vocab_size, self.width = embed.shape
        if head is None:
            head = embed
        if tuple(head.shape) != (self.vocab_size, self.width):
            raise ValueError(f"head of shape {tuple(head.shape)}, expected {(self.vocab_size, self.width)}")
        self.streams, self.eps, self.dtype = int(streams), float(eps), dtype
        self.max_seq, self.max_batch = max_seq, max_batch
        self.max_rows = max_rows or min(max_seq, 512) * max_batch
        self._tensors = []
        self.embed_scale = float(embed_scale)
        self._head = self._keep(pack_matrix([head], 256))
        # (a head that is the table itself is one matrix where the strides allow)
        self._embed = self._head if head is embed and self.width % 256 == 0 else self._keep(pack_matrix([embed]))
        self._final_norm = self._keep(pack_vector(final_norm, 64))
        self._final_norm_b = None if final_norm_b is None else self._keep(pack_vector(final_norm_b, 64))
        self.specs = list(layers)
        self.runs = plan_runs(self.specs, order)
        self._layers = [self._pack_layer(s) for s in layers]
        self._handle = None
        for s in self.specs:      # the packed copies are the weights from here on
            s.q = s.k = s.v = s.o = s.gate = s.up = s.down = s.experts = None
            if s.latent is not None:
                s.latent.dq = s.latent.uq = s.latent.dkv = s.latent.uk = s.latent.uv = s.latent.gate = None

    def _keep(self, t):
        self._tensors.append(t)
        return t

    def _put(self, t):
        return ptr(self._keep(t))

    def _pack_layer(self, s: LayerSpec):
        put = self._put
        ff = 0 if s.gate is None else s.gate.shape[0]
        if s.experts is not None:
            ff = s.experts.gate[0].shape[0]
        c = abi.DecoderLayer(heads=s.heads, kv_heads=s.kv_heads, dim=s.dim, vdim=s.vdim, unit_qk=int(s.unit_qk),
                             chunk=int(s.chunk), window=int(s.window), ff=ff, scale=float(s.scale), parallel=int(s.parallel),
                             act=ACTIVATIONS[s.act])
        if s.latent is not None:
            self._pack_latent(c, s)
        else:
            self._pack_heads(c, s)
        c.norm1 = put(pack_vector(s.norm1, 64))
        if s.norm1_b is not None:
            c.norm1_b = put(pack_vector(s.norm1_b, 64))
        if s.sinks is not None:
            if s.sinks.numel() != s.heads:
                raise ValueError("one sink per query head is needed")
            c.sinks = put(pack_vector(s.sinks))
        if ff:
            if s.experts is not None:
                self._pack_experts(c, s.experts, ff)
            else:
                if tuple(s.gate.shape) != (ff, self.width) or tuple(s.up.shape) != (ff, self.width) or \
                        tuple(s.down.shape) != (self.width, ff):
                    raise ValueError("feed-forward matrices do not fit together")
                c.gate_up = put(pack_matrix([s.gate, s.up]))
                c.down = put(pack_matrix([s.down]))
            c.norm2 = put(pack_vector(s.norm2, 64))
            if s.norm2_b is not None:
                c.norm2_b = put(pack_vector(s.norm2_b, 64))
        if s.parallel and self.streams != 1:
            raise ValueError("sublayers that read the same residual need one stream")
        self._pack_connections(c, s, ff)
        return c

    def _pack_heads(self, c, s: LayerSpec):
        torch = abi.require_cuda()
        if s.heads % s.kv_heads:
            raise ValueError(f"{s.heads} query heads cannot share {s.kv_heads} key/value heads evenly")
        for name, t, shape in (("q", s.q, (s.heads * s.dim, self.width)), ("k", s.k, (s.kv_heads * s.dim, self.width)),
                               ("v", s.v, (s.kv_heads * s.vdim, self.width)), ("o", s.o, (self.width, s.heads * s.vdim))):
            expect(name, t, shape)
        c.qkv = self._put(pack_matrix([s.q, s.k, s.v]))
        c.o = self._put(pack_matrix([s.o]))
        if s.slopes is not None:
            if len(s.slopes) != s.heads:
                raise ValueError("one distance-bias slope per query head is needed")
            c.slopes = self._put(pack_vector(torch.tensor(list(s.slopes), dtype=torch.float64)))

    def _pack_latent(self, c, s: LayerSpec):
        """Heads, latents and rotated parts padded to the row layout the kernels read."""
        a, put = s.latent, self._put
        h, dp, vp = s.heads, _round(s.dim, 8), _round(s.vdim, 8)
        rp, kp = _round(a.rot_dim, 16), _round(a.rank, 16)
        expect("uk", a.uk, (h * s.dim, a.rank))
        expect("uv", a.uv, (h * s.vdim, a.rank))
        expect("o", s.o, (self.width, h * s.vdim))
        c.mixer, c.kv_rank, c.rot_dim, c.q_rank = abi.MIXER_LATENT, a.rank, a.rot_dim, 0
        c.own_kv, c.gated = int(a.dkv is not None), int(a.gate is not None)
        if a.rot_dim % 2:
            raise ValueError(f"rotated part of {a.rot_dim} columns: pairs are needed")

        def query_rows(q, inn):
            expect("q", q, (h * (s.dim + a.rot_dim), inn))
            q = q.reshape(h, s.dim + a.rot_dim, inn)
            rows = q.new_zeros((h, dp + rp, inn))
            rows[:, :s.dim], rows[:, dp:dp + a.rot_dim] = q[:, :s.dim], q[:, s.dim:]
            return rows.reshape(h * (dp + rp), inn)

        if a.dq is not None:
            c.q_rank = a.dq.shape[0]
            expect("dq", a.dq, (c.q_rank, self.width))
            parts = [pad_rows(a.dq, _round(c.q_rank, 16))]
            c.uq, c.q_norm = put(pack_matrix([query_rows(a.uq, c.q_rank)])), put(pack_vector(a.q_norm, 64))
        else:
            parts = [query_rows(s.q, self.width)]
        if a.dkv is not None:
            expect("dkv", a.dkv, (a.rank + a.rot_dim, self.width))
            parts += [pad_rows(a.dkv[:a.rank], kp), pad_rows(a.dkv[a.rank:], rp)]
            c.kv_norm = put(pack_vector(a.kv_norm, 64))
        if a.gate is not None:
            expect("gate", a.gate, (h, self.width))
            parts.append(a.gate)
        c.in_proj = put(pack_matrix(parts))
        uk, uv = a.uk.reshape(h, s.dim, a.rank), a.uv.reshape(h, s.vdim, a.rank)
        keys, values = uk.new_zeros((h, dp, a.rank)), uv.new_zeros((h, vp, a.rank))
        keys[:, :s.dim], values[:, :s.vdim] = uk, uv
        c.uk_uv = put(pack_matrix([keys.reshape(h * dp, a.rank), values.reshape(h * vp, a.rank)]))
        turned = uk.new_zeros((h, kp, s.dim))
        turned[:, :a.rank] = uk.transpose(1, 2)
        c.uk_t = put(pack_matrix([turned.reshape(h * kp, s.dim)]))
        o = s.o.new_zeros((self.width, h, vp))
        o[:, :, :s.vdim] = s.o.reshape(self.width, h, s.vdim)
        c.o = put(pack_matrix([o.reshape(self.width, h * vp)]))

    def _pack_experts(self, c, e: Experts, ff):
        n = len(e.gate)
        if not (0 < e.top <= n == len(e.up) == len(e.down)):
            raise ValueError(f"{e.top} of {n} experts, {len(e.up)} up and {len(e.down)} down matrices")
        for g, u, d in zip(e.gate, e.up, e.down):
            expect("expert gate", g, (ff, self.width))
            expect("expert up", u, (ff, self.width))
            expect("expert down", d, (self.width, ff))
        expect("router", e.router, (n, self.width))
        c.experts, c.top = n, e.top
        c.gate_up = self._put(pack_matrix([t for g, u in zip(e.gate, e.up) for t in (g, u)]))
        c.down = self._put(pack_matrix(list(e.down)))
        c.router = self._put(pack_matrix([e.router]))
        if e.bias is not None:
            c.router_b = self._put(pack_vector(e.bias))

    def _pack_connections(self, c, s: LayerSpec, ff):
        torch = abi.require_cuda()
        for q, hc in ((1, s.hc1), (2, s.hc2)):
            if q == 2 and not ff:
                continue
            if hc is None:
                if self.streams != 1:
                    raise ValueError("several streams need connections in every sublayer")
                one = torch.ones(1)
                hc = Connections(one, one, one.reshape(1, 1))
            if tuple(hc.mix.shape) != (self.streams, self.streams) or hc.in_.numel() != self.streams or \
                    hc.out.numel() != self.streams:
                raise ValueError("connection tensors do not fit the number of streams")
            setattr(c, f"hc{q}_in", self._put(pack_vector(hc.in_)))
            setattr(c, f"hc{q}_out", self._put(pack_vector(hc.out)))
            setattr(c, f"hc{q}_mix", self._put(pack_vector(hc.mix)))

    # -- caches and handle -----------------------------------------------------------------
    def _grow_cache(self, run, max_batch, max_seq):
        torch = abi.require_cuda()
        s = self.specs[run.layer]
        if run.source is not None:      # (the source runs first: its caches are grown)
            run.k_cache, run.v_cache = run.source.k_cache, run.source.v_cache
            return
        old = run.k_cache
        if old is not None and old.shape[0] >= max_batch and old.shape[2] >= max_seq:
            if tuple(old.shape[:3:2]) == (max_batch, max_seq):
                return
        dt = torch.float32 if self.dtype == "float32" else torch.bfloat16
        if s.latent is not None:        # one row per position: latent and rotated key part
            kinds = (("k_cache", 1, _round(s.latent.rank, 16) + _round(s.latent.rot_dim, 16)),)
        else:
            kinds = (("k_cache", s.kv_heads, _round(s.dim, 8)), ("v_cache", s.kv_heads, _round(s.vdim, 8)))
        for name, heads, d in kinds:
            new = torch.zeros((max_batch, heads, max_seq, d), dtype=dt, device="cuda")
            prev = getattr(run, name)
            if prev is not None:
                new[:prev.shape[0], :, :prev.shape[2]] = prev
            setattr(run, name, new)

    def _ensure_handle(self, batch=1, seq=1, total=1):
        h = self._handle
        if h is None or batch > h.cfg.max_batch or total > h.cfg.max_seq or batch * seq > h.cfg.max_rows:
            self.max_batch = max(self.max_batch, batch)
            self.max_seq = max(self.max_seq, total)
            self.max_rows = max(self.max_rows, batch * seq)
            self._handle = None
            self._handle = _DecoderHandle(self, self.max_batch, self.max_seq, self.max_rows)
        return self._handle

    def _caches(self, length, batch):
        return [KVCache(run, length, batch) for run in self.runs]
