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


@dataclass
class Connections:
    """Hyper-connection of one sublayer: ``in_`` [streams], ``out`` [streams], ``mix`` [from, to].  None in a
    LayerSpec is the ordinary residual (one stream)."""
    in_: object
    out: object
    mix: object


@dataclass
class LayerSpec:
    """One layer.  Matrices are [out, in] torch tensors.  ``slopes``: distance-bias slope per query head, or
    None; ``chunk``: chunk length of the mask, or 0; ``gate`` None: no feed-forward."""
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


class _Run:
    """One run of a layer: owner of its caches."""

    def __init__(self, layer):
        self.layer = layer
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
                                     max_seq=max_seq, max_rows=max_rows)
        layers = (abi.DecoderLayer * len(model._layers))(*model._layers)
        runs = (abi.DecoderRun * len(model.runs))()
        for r, run in zip(runs, model.runs):
            r.layer, r.k_cache, r.v_cache = run.layer, ptr(run.k_cache), ptr(run.v_cache)
        need = lib.rotor_b200_decoder_workspace_bytes(C.byref(self.cfg), layers)
        if need == 0:
            raise RotorB200Error("decoder shape not supported by the GPU path (width up to 10240, up to 16 streams, "
                                 "head sizes up to 512)")
        self.workspace = torch.empty(need, dtype=torch.uint8, device="cuda")
        self.keep = (model._tensors, [(r.k_cache, r.v_cache) for r in model.runs])  # the handle points into these
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
    """``order``: layer index of every run, in the order they run."""

    def __init__(self, layers: Sequence[LayerSpec], order: Sequence[int], embed, head, final_norm, *, streams: int = 1,
                 eps: float = 1e-6, dtype: str = "bfloat16", max_seq: int = 2048, max_batch: int = 1,
                 max_rows: Optional[int] = None):
        torch = abi.require_cuda()
        if dtype not in DTYPES:
            raise ValueError(f"dtype {dtype!r} is not one of {DTYPES}")
        if not layers or not order:
            raise ValueError("a decoder needs at least one layer and one run")
        self.vocab_size, self.width = embed.shape
        if tuple(head.shape) != (self.vocab_size, self.width):
            raise ValueError(f"head of shape {tuple(head.shape)}, expected {(self.vocab_size, self.width)}")
        self.streams, self.eps, self.dtype = int(streams), float(eps), dtype
        self.max_seq, self.max_batch = max_seq, max_batch
        self.max_rows = max_rows or min(max_seq, 512) * max_batch
        self._tensors = []
        self._embed = self._keep(pack_matrix([embed]))
        self._head = self._keep(pack_matrix([head], 256))
        self._final_norm = self._keep(pack_vector(final_norm, 64))
        self.specs = list(layers)
        self._layers = [self._pack_layer(s) for s in layers]
        self.runs = [_Run(int(i)) for i in order]
        for r in self.runs:
            if not 0 <= r.layer < len(layers):
                raise ValueError(f"run of layer {r.layer}, but there are {len(layers)} layers")
        self._handle = None
        for s in self.specs:      # the packed copies are the weights from here on
            s.q = s.k = s.v = s.o = s.gate = s.up = s.down = None

    def _keep(self, t):
        self._tensors.append(t)
        return t

    def _pack_layer(self, s: LayerSpec):
        torch = abi.require_cuda()
        if s.heads % s.kv_heads:
            raise ValueError(f"{s.heads} query heads cannot share {s.kv_heads} key/value heads evenly")
        for name, t, shape in (("q", s.q, (s.heads * s.dim, self.width)), ("k", s.k, (s.kv_heads * s.dim, self.width)),
                               ("v", s.v, (s.kv_heads * s.vdim, self.width)), ("o", s.o, (self.width, s.heads * s.vdim))):
            if tuple(t.shape) != shape:
                raise ValueError(f"{name} projection of shape {tuple(t.shape)}, expected {shape}")
        ff = 0 if s.gate is None else s.gate.shape[0]
        if ff and (tuple(s.gate.shape) != (ff, self.width) or tuple(s.up.shape) != (ff, self.width) or
                   tuple(s.down.shape) != (self.width, ff)):
            raise ValueError("feed-forward matrices do not fit together")
        c = abi.DecoderLayer(heads=s.heads, kv_heads=s.kv_heads, dim=s.dim, vdim=s.vdim, unit_qk=int(s.unit_qk),
                             chunk=int(s.chunk), ff=ff, scale=float(s.scale))
        put = lambda t: ptr(self._keep(t))
        c.qkv = put(pack_matrix([s.q, s.k, s.v]))
        c.o = put(pack_matrix([s.o]))
        c.norm1 = put(pack_vector(s.norm1, 64))
        if s.slopes is not None:
            if len(s.slopes) != s.heads:
                raise ValueError("one distance-bias slope per query head is needed")
            c.slopes = put(pack_vector(torch.tensor(list(s.slopes), dtype=torch.float64)))
        if ff:
            c.gate_up = put(pack_matrix([s.gate, s.up]))
            c.down = put(pack_matrix([s.down]))
            c.norm2 = put(pack_vector(s.norm2, 64))
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
            setattr(c, f"hc{q}_in", put(pack_vector(hc.in_)))
            setattr(c, f"hc{q}_out", put(pack_vector(hc.out)))
            setattr(c, f"hc{q}_mix", put(pack_vector(hc.mix)))
        return c

    # -- caches and handle -----------------------------------------------------------------
    def _grow_cache(self, run, max_batch, max_seq):
        torch = abi.require_cuda()
        s = self.specs[run.layer]
        old = run.k_cache
        if old is not None and old.shape[0] >= max_batch and old.shape[2] >= max_seq:
            if tuple(old.shape[:3:2]) == (max_batch, max_seq):
                return
        dt = torch.float32 if self.dtype == "float32" else torch.bfloat16
        for name, d in (("k_cache", s.dim), ("v_cache", s.vdim)):
            new = torch.zeros((max_batch, s.kv_heads, max_seq, _round(d, 8)), dtype=dt, device="cuda")
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
