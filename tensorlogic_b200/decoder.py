"""Config-driven decoder: dense bf16 / f32 weights, layers described one by one.

    DecoderArch / LayerArch / LatentLayerArch
                              sizes and constants of a model, read by its design's module
    Decoder                   the runner (tlc_decoder_* of include/tlcuda.h): sequences with cache
                              slots, portions of prompts, greedy or temperature decoding
    load_safetensors          a safetensors file -> Model

Weights stay in HBM; nothing here computes on the host.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from typing import Optional, Sequence

import numpy as np

from . import _lib, synth
from ._lib import DecoderConfig, DecoderLayer, TensorError, check
from .api import Device, QTensor
from .model import Model

DTYPES = {"bfloat16": _lib.TYPE_BF16, "float32": _lib.TYPE_F32}


@dataclass
class LayerArch:
    """One layer: grouped-query attention over a sliding window with kept first tokens, values = keys,
    and a feed-forward (``ff_kind``: "none", "clamped_glu" or "moe")."""
    heads: int
    kv_heads: int
    dim: int
    window: int
    keep_first: int
    rot_dims: int
    rot_base: float
    scale: float
    ff_kind: str = "none"
    ff: int = 0
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    expert_ff: int = 0
    shared_ff: int = 0

    def struct(self) -> DecoderLayer:
        kind = {"none": _lib.FF_NONE, "clamped_glu": _lib.FF_CLAMPED_GLU, "moe": _lib.FF_MOE}[self.ff_kind]
        return DecoderLayer(self.heads, self.kv_heads, self.dim, min(self.window, 2**31 - 1), self.keep_first, self.rot_dims,
                            self.rot_base, self.scale, kind, self.ff, self.limit, self.experts, self.top, self.expert_ff,
                            self.shared_ff, _lib.MIX_WINDOW)

    def tensor_shapes(self, p: str, w: int, _streams: int) -> dict:
        q, k = self.heads * self.dim, self.kv_heads * self.dim
        out = {p + "norm1": (1, w), p + "mix.q": (q, w), p + "mix.q.b": (1, q), p + "mix.q.norm": (1, q), p + "mix.k": (k, w),
               p + "mix.k.b": (1, k), p + "mix.k.norm": (1, k), p + "mix.o": (w, q), p + "mix.o.b": (1, w)}
        if self.ff_kind != "none":
            out[p + "norm2"] = (1, w)

        def glu(at, n):
            out.update({at + "gate": (n, w), at + "up": (n, w), at + "down": (w, n)})
        if self.ff_kind == "clamped_glu":
            glu(p + "mlp.", self.ff)
        elif self.ff_kind == "moe":
            out[p + "mlp.router"] = (self.experts, w)
            for e in range(self.experts):
                glu(f"{p}mlp.e{e}.", self.expert_ff)
            if self.shared_ff:
                glu(p + "mlp.shared.", self.shared_ff)
                out[p + "mlp.shared.sg"] = (1, w)
        return out


@dataclass
class LatentLayerArch:
    """One layer over several residual streams: latent attention (``dim`` unrotated and ``rot_dim`` rotated
    entries per head and key, ``vdim`` per value) and a feed-forward (``ff_kind``: "none" or "silu_glu")."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    rot_base: float
    scale: float
    ff_kind: str = "none"
    ff: int = 0

    def struct(self) -> DecoderLayer:
        kind = {"none": _lib.FF_NONE, "silu_glu": _lib.FF_SILU_GLU}[self.ff_kind]
        return DecoderLayer(heads=self.heads, dim=self.dim, rot_dims=self.rot_dim, rot_base=self.rot_base, scale=self.scale,
                            ff_kind=kind, ff=self.ff, mixer=_lib.MIX_LATENT, vdim=self.vdim, q_rank=self.q_rank, kv_rank=self.kv_rank)

    def tensor_shapes(self, p: str, w: int, streams: int) -> dict:
        h, m = self.heads, p + "mix."
        out = {m + "dq": (self.q_rank, w), m + "dq.norm": (1, self.q_rank), m + "uq": (h * (self.dim + self.rot_dim), self.q_rank),
               m + "dkv": (self.kv_rank + self.rot_dim, w), m + "dkv.norm": (1, self.kv_rank), m + "uk": (h * self.dim, self.kv_rank),
               m + "uv": (h * self.vdim, self.kv_rank), m + "sink": (1, h), m + "o": (w, h * self.vdim)}
        for q in (1, 2) if self.ff_kind != "none" else (1,):
            out.update({f"{p}norm{q}": (1, w), f"{p}norm{q}.b": (1, w), f"{p}norm{q}.alpha": (1, 1), f"{p}ls{q}": (1, w),
                        f"{p}hc{q}.in": (1, streams), f"{p}hc{q}.out": (1, streams), f"{p}hc{q}.mix": (streams, streams)})
        if self.ff_kind != "none":
            f = p + "mlp."
            out.update({f + "gate": (self.ff, w), f + "gate.b": (1, self.ff), f + "up": (self.ff, w), f + "up.b": (1, self.ff),
                        f + "down": (w, self.ff), f + "down.b": (1, w)})
        return out

    def weight_bytes(self, w: int, elem: int = 2) -> int:
        """Bytes of the matrices one token uses."""
        h = self.heads
        n = self.q_rank * (w + h * (self.dim + self.rot_dim)) + w * (self.kv_rank + self.rot_dim) + \
            h * (self.dim + self.vdim) * self.kv_rank + w * h * self.vdim + (3 * w * self.ff if self.ff_kind != "none" else 0)
        return n * elem


@dataclass
class DecoderArch:
    width: int
    vocab: int
    norm_eps: float
    layers: list = field(default_factory=list)   # LayerArch, or LatentLayerArch with streams > 0
    streams: int = 0                             # residual streams; 0: one residual, parallel branches
    logit_softcap: float = 0.0
    runs: Optional[list[int]] = None             # layer numbers in the order they run (None: each once)

    def tensor_shapes(self) -> dict:
        """Tensor names -> (rows, cols) as tlc_decoder_create binds them."""
        out = {"embed": (self.vocab, self.width), "final.norm": (1, self.width)}
        if self.streams:
            out.update({"final.norm.b": (1, self.width), "final.norm.alpha": (1, 1)})
        for i, l in enumerate(self.layers):
            out.update(l.tensor_shapes(f"l{i}.", self.width, self.streams))
        return out

    def layer_weight_bytes(self, l, elem: int = 2, active_only: bool = True) -> int:
        """Bytes of the matrices one token uses in layer ``l`` (all experts with active_only=False)."""
        if isinstance(l, LatentLayerArch):
            return l.weight_bytes(self.width, elem)
        w, q, k = self.width, l.heads * l.dim, l.kv_heads * l.dim
        n = w * (q + k) + q * w
        if l.ff_kind == "clamped_glu":
            n += 3 * w * l.ff
        elif l.ff_kind == "moe":
            n += w * l.experts + 3 * w * l.expert_ff * (l.top if active_only else l.experts) + 3 * w * l.shared_ff
        return n * elem


def load_safetensors(dev: Device, path, dtype: str = "bfloat16") -> Model:
    h = C.c_void_p()
    check(dev.lib.tlc_model_load_safetensors(dev.handle, str(path).encode(), DTYPES[dtype], C.byref(h)))
    return Model(dev, h)


def dense_tensor(dev: Device, array, dtype: str = "bfloat16") -> QTensor:
    """A float array as a resident bf16 / f32 weight."""
    a = np.ascontiguousarray(array, np.float32)
    rows, cols = (1, a.size) if a.ndim <= 1 else (int(np.prod(a.shape[:-1])), a.shape[-1])
    h = C.c_void_p()
    check(dev.lib.tlc_qtensor_create_dense(dev.handle, _lib.TYPE_F32, DTYPES[dtype], rows, cols, a.ctypes.data, a.nbytes,
                                           C.byref(h)))
    return QTensor(dev, h)


def model_from_arrays(dev: Device, weights: dict, dtype: str = "bfloat16") -> Model:
    m = Model(dev)
    for name, a in weights.items():
        m.add(name, dense_tensor(dev, a, dtype))
    return m


def synthetic_decoder(dev: Device, arch: DecoderArch, seed: int, dtype: str = "bfloat16") -> Model:
    """Random weights made on the device: matrices N(0, 1/columns), norm weights and scales N(1, 0.02), biases
    N(0, 0.02), coefficients of n streams N(1 / n, 0.02)."""
    m = Model(dev)
    for name, (rows, cols) in arch.tensor_shapes().items():
        last = name.rsplit(".", 1)[-1]
        mean, std = ((1.0 / cols, 0.02) if last in ("alpha", "mix", "in", "out") else
                     (0.0, 0.02) if last in ("b", "sink") else (1.0, 0.02) if "norm" in name or last in ("ls1", "ls2") else
                     (0.0, cols ** -0.5))
        h = C.c_void_p()
        check(dev.lib.tlc_qtensor_create_normal_dense(dev.handle, DTYPES[dtype], rows, cols, seed, synth.tensor_id(name), mean,
                                                      std, C.byref(h)))
        m.add(name, QTensor(dev, h))
    return m


def _ints(a):
    return a.ctypes.data_as(C.POINTER(C.c_int32))


class Decoder:
    """Runner over a Model.  Sequences occupy cache slots 0 .. max_batch - 1; ``open`` hands out a free
    one, ``close`` gives it back.  ``prefill`` and ``decode`` mirror the Llama runner's."""

    dtypes = tuple(DTYPES)

    def __init__(self, dev: Device, model: Model, arch: DecoderArch, dtype: str = "bfloat16", max_seq: int = 2048,
                 max_batch: int = 1, max_prefill: int = 2048, max_logit_rows: Optional[int] = None, use_graph: bool = True):
        self.dev, self.model, self.arch, self.dtype = dev, model, arch, dtype
        self.max_seq, self.max_batch = max_seq, max_batch
        max_prefill = max(1, min(max_prefill, max_seq))
        if max_logit_rows is None:  # up to 256 MiB of logits
            max_logit_rows = max(1, min(max_prefill, (256 << 20) // (4 * arch.vocab)))
        layers = (DecoderLayer * len(arch.layers))(*[l.struct() for l in arch.layers])
        runs = np.ascontiguousarray(arch.runs if arch.runs is not None else range(len(arch.layers)), np.int32)
        cfg = DecoderConfig(len(arch.layers), arch.width, arch.vocab, arch.norm_eps, DTYPES[dtype], max_seq, max_batch,
                            max_prefill, max_logit_rows, int(not use_graph), arch.streams, arch.logit_softcap,
                            runs.size, layers, _ints(runs))
        h = C.c_void_p()
        check(dev.lib.tlc_decoder_create(dev.handle, model.handle, C.byref(cfg), C.byref(h)))
        self.handle = h
        self._free = list(range(max_batch - 1, -1, -1))
        self._length = [0] * max_batch

    def __del__(self):
        try:
            if self.handle and self.dev.handle:
                self.dev.lib.tlc_decoder_destroy(self.handle)
            self.handle = None
        except Exception:
            pass

    # -- sequences ---------------------------------------------------------
    def open(self) -> int:
        if not self._free:
            raise TensorError(_lib.ERR_BUFFER_EXHAUSTED, f"all {self.max_batch} sequences are in use")
        return self._free.pop()

    def close(self, seq: int) -> None:
        check(self.dev.lib.tlc_decoder_release(self.handle, seq))
        self._length[seq] = 0
        self._free.append(seq)

    def length(self, seq: int) -> int:
        return self._length[seq]

    def feed(self, seq: int, tokens, want: Sequence[int] = ()) -> np.ndarray:
        """The sequence's next tokens; returns the f32 logits [len(want), vocab] at the wanted places."""
        tokens = np.ascontiguousarray(tokens, np.int32).reshape(-1)
        if tokens.size == 1 and seq == 0 and self._length[0] > 0:
            _, logits = self.decode(tokens, return_logits=True)  # the step a generation makes
            return logits[:len(want)]
        return self.prefill(tokens, self._length[seq], seq=seq, want=want, sample=False)[1]

    # -- the calls the Llama runner has -------------------------------------
    def prefill(self, ids, pos0: int = 0, return_logits: bool = True, all_rows: bool = False, seq: int = 0,
                want: Optional[Sequence[int]] = None, sample: bool = True):
        """Returns (next token or None, f32 logits [rows, vocab] or None): of the last row, of all rows, or
        of the places in ``want``."""
        ids = np.ascontiguousarray(ids, np.int32).reshape(-1)
        if want is None:
            want = range(ids.size) if all_rows else [ids.size - 1] if return_logits else []
        order = np.ascontiguousarray(sorted(set(int(w) for w in want)), np.int32)
        logits = np.empty((order.size, self.arch.vocab), np.float32)
        nxt = C.c_int32()
        check(self.dev.lib.tlc_decoder_prefill(self.handle, seq, _ints(ids), ids.size, pos0, _ints(order), order.size,
                                               logits.ctypes.data_as(C.POINTER(C.c_float)), C.byref(nxt) if sample else None))
        self._length[seq] = pos0 + ids.size
        if list(order) != list(want):
            at = {int(p): i for i, p in enumerate(order)}
            logits = logits[[at[int(p)] for p in want]]
        return (nxt.value if sample else None), (logits if return_logits else None)

    def set_sampling(self, temperature: float = 0.0, seed: int = 0) -> None:
        check(self.dev.lib.tlc_decoder_set_sampling(self.handle, float(temperature), int(seed)))

    def set_state(self, ids, positions) -> None:
        ids = np.ascontiguousarray(ids, np.int32).reshape(-1)
        pos = np.ascontiguousarray(positions, np.int32).reshape(-1)
        if ids.size != pos.size:
            raise TensorError(_lib.ERR_SHAPE_MISMATCH, "ids and positions differ in length")
        check(self.dev.lib.tlc_decoder_set_state(self.handle, ids.size, _ints(ids), _ints(pos)))
        self._length[:ids.size] = [int(p) for p in pos]

    def decode(self, ids=None, batch: int = 1, return_logits: bool = False):
        """One step of sequences 0 .. batch - 1 through host buffers.  Returns (next tokens, logits or None)."""
        if ids is not None:
            ids = np.ascontiguousarray(ids, np.int32).reshape(-1)
            batch = ids.size
        nxt = np.empty(batch, np.int32)
        logits = np.empty((batch, self.arch.vocab), np.float32) if return_logits else None
        check(self.dev.lib.tlc_decoder_decode_host(self.handle, batch, _ints(ids) if ids is not None else None, _ints(nxt),
                                                   logits.ctypes.data_as(C.POINTER(C.c_float)) if return_logits else None))
        for i in range(batch):
            self._length[i] += 1
        return nxt, logits

    def decode_enqueue(self, batch: int, steps: int) -> None:
        check(self.dev.lib.tlc_decoder_decode_enqueue(self.handle, batch, steps))
        for i in range(batch):
            self._length[i] += steps

    def read_state(self, batch: int = 1):
        nxt, pos = np.empty(batch, np.int32), np.empty(batch, np.int32)
        check(self.dev.lib.tlc_decoder_read_state(self.handle, batch, _ints(nxt), _ints(pos)))
        return nxt, pos

    @property
    def launches_per_step(self) -> int:
        return int(self.dev.lib.tlc_decoder_launches_per_step(self.handle))
