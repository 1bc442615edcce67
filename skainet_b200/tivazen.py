"""Host-side configuration, loader and handle of the Tivazen design (include/skainet_cuda_tivazen.h): every size and constant
comes from config.json, every matrix from model.safetensors (BF16, [out, in])."""
from __future__ import annotations

import ctypes as C
import json
import os
from dataclasses import dataclass
from typing import Any, Dict, List, Optional

import numpy as np

from . import _lib as L
from .decoder import Decoder
from .device import Weight
from .safetensors import SafetensorsReader

MLP_NONE, MLP_DENSE, MLP_MOE = 0, 1, 2
W_EMBED, W_HEAD, W_Q, W_DKV, W_UK, W_UV, W_G, W_O, W_ROUTER, W_GATE, W_UP, W_DOWN = range(12)
V_NORM1, V_NORM2, V_DKV_NORM, V_DEPTH, V_FINAL_NORM = range(5)


class _Layer(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "kv_from", "window")] + \
               [("scale", C.c_float), ("rope_base", C.c_double)] + \
               [(n, C.c_int32) for n in ("mlp", "ff", "experts", "top")]


class _Config(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("n_layers", "width", "vocab")] + [("eps", C.c_float)] + \
               [(n, C.c_int32) for n in ("max_seq", "max_batch", "prefill_rows", "act_f32")]


def _only(d: Dict[str, Any], what: str, *keys: str) -> None:
    extra = sorted(set(d) - set(keys))
    if extra:
        raise ValueError(f"Tivazen: {what} has unknown keys {extra}")


@dataclass
class TivazenLayer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    window: int
    scale: float
    rope_base: float
    kv_from: Optional[int] = None
    mlp: int = MLP_NONE
    ff: int = 0
    experts: int = 0
    top: int = 0

    @classmethod
    def from_json(cls, d: Dict[str, Any], index: int) -> "TivazenLayer":
        what = f"layer {index}"
        _only(d, what, "type", "mixer", "mlp")
        if d["type"] != "latent_attention":
            raise ValueError(f"Tivazen: {what}: mixer type {d['type']!r} not supported")
        m = d["mixer"]
        _only(m, what + " mixer", "heads", "dim", "rot_dim", "vdim", "kv_rank", "kv_from", "mask", "rot", "scale")
        _only(m["mask"], what + " mask", "size")
        _only(m["rot"], what + " rot", "base", "dims")
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError(f"Tivazen: {what}: rotation of {m['rot']['dims']} dimensions, rot_dim {m['rot_dim']}")
        out = cls(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["mask"]["size"], float(m["scale"]), float(m["rot"]["base"]), m.get("kv_from"))
        f = d.get("mlp")
        if f is None:
            return out
        if f["kind"] == "dense":
            _only(f, what + " mlp", "kind", "ff")
            out.mlp, out.ff = MLP_DENSE, f["ff"]
        elif f["kind"] == "moe":
            _only(f, what + " mlp", "kind", "expert", "router")
            _only(f["expert"], what + " expert", "ff")
            _only(f["router"], what + " router", "experts", "top")
            out.mlp, out.ff, out.experts, out.top = MLP_MOE, f["expert"]["ff"], f["router"]["experts"], f["router"]["top"]
        else:
            raise ValueError(f"Tivazen: {what}: feed-forward kind {f['kind']!r} not supported")
        return out

    def to_c(self) -> _Layer:
        return _Layer(self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank, -1 if self.kv_from is None else self.kv_from, self.window,
                      self.scale, self.rope_base, self.mlp, self.ff, self.experts, self.top)


@dataclass
class TivazenConfig:
    width: int
    vocab: int
    eps: float
    layers: List[TivazenLayer]
    max_seq: int = 1024
    max_batch: int = 1
    prefill_rows: int = 0            # rows of one prompt pass, 0: the library's choice
    dtype: str = "bfloat16"          # or "float32": activations, cache and arithmetic in 32-bit

    @classmethod
    def from_json(cls, d: Dict[str, Any], **runtime) -> "TivazenConfig":
        _only(d, "config", "architecture", "layers", "norm", "vocab", "width")
        _only(d["norm"], "norm", "eps")
        return cls(d["width"], d["vocab"], float(d["norm"]["eps"]), [TivazenLayer.from_json(l, i) for i, l in enumerate(d["layers"])], **runtime)

    def to_c(self):
        if self.dtype not in ("bfloat16", "float32"):
            raise ValueError(f"Tivazen: dtype {self.dtype!r} is neither bfloat16 nor float32")
        c = _Config(len(self.layers), self.width, self.vocab, self.eps, self.max_seq, self.max_batch, self.prefill_rows, int(self.dtype == "float32"))
        return c, (_Layer * len(self.layers))(*[l.to_c() for l in self.layers])


class Tivazen(Decoder):
    architecture = "Tivazen"

    def __init__(self, cfg: TivazenConfig):
        self.cfg = cfg
        h = C.c_int64()
        c, layers = cfg.to_c()
        L.check(L.lib().skainet_cuda_tivazen_create(C.byref(c), layers, C.byref(h)))
        super().__init__(h.value, cfg.vocab, cfg.max_seq, cfg.max_batch)

    # ---- weights --------------------------------------------------------------------------------
    def set_weight(self, layer: int, which: int, w: Weight, expert: int = 0) -> None:
        """Copies w into the model."""
        L.check(L.lib().skainet_cuda_tivazen_set_weight(self.handle, layer, which, expert, w.handle))

    def set_vector(self, layer: int, which: int, values) -> None:
        v = np.ascontiguousarray(values, dtype=np.float32).reshape(-1)
        L.check(L.lib().skainet_cuda_tivazen_set_vector(self.handle, layer, which, v.ctypes.data_as(L.f32p), v.size))

    def synth(self, seed: int = 100, std: float = 0.02) -> None:
        L.check(L.lib().skainet_cuda_tivazen_synth(self.handle, seed, std))

    def load(self, r: SafetensorsReader) -> None:
        cfg = self.cfg

        def matrix(layer: int, which: int, name: str, rows: int, cols: int, expert: int = 0) -> None:
            w = r.weight(name, rows, cols)
            self.set_weight(layer, which, w, expert)
            w.free()

        matrix(0, W_EMBED, "embed", cfg.vocab, cfg.width)
        matrix(0, W_HEAD, "head", cfg.vocab, cfg.width)
        self.set_vector(0, V_FINAL_NORM, r.floats("final.norm"))
        for i, l in enumerate(cfg.layers):
            p = f"l{i}."
            matrix(i, W_Q, p + "mix.q", l.heads * (l.dim + l.rot_dim), cfg.width)
            matrix(i, W_UK, p + "mix.uk", l.heads * l.dim, l.kv_rank)
            matrix(i, W_UV, p + "mix.uv", l.heads * l.vdim, l.kv_rank)
            matrix(i, W_G, p + "mix.g", l.heads, cfg.width)
            matrix(i, W_O, p + "mix.o", cfg.width, l.heads * l.vdim)
            if l.kv_from is None:
                matrix(i, W_DKV, p + "mix.dkv", l.kv_rank + l.rot_dim, cfg.width)
                self.set_vector(i, V_DKV_NORM, r.floats(p + "mix.dkv.norm"))
            self.set_vector(i, V_NORM1, r.floats(p + "norm1"))
            self.set_vector(i, V_DEPTH, r.floats(p + "dwa"))
            if l.mlp == MLP_NONE:
                continue
            self.set_vector(i, V_NORM2, r.floats(p + "norm2"))
            if l.mlp == MLP_MOE:
                matrix(i, W_ROUTER, p + "mlp.router", l.experts, cfg.width)
            for e in range(l.experts if l.mlp == MLP_MOE else 1):
                q = p + (f"mlp.e{e}." if l.mlp == MLP_MOE else "mlp.")
                matrix(i, W_GATE, q + "gate", l.ff, cfg.width, e)
                matrix(i, W_UP, q + "up", l.ff, cfg.width, e)
                matrix(i, W_DOWN, q + "down", cfg.width, l.ff, e)

    @classmethod
    def from_dir(cls, path: str, config: Optional[Dict[str, Any]] = None, **runtime) -> "Tivazen":
        """The model of a folder with config.json and model.safetensors."""
        if config is None:
            with open(os.path.join(path, "config.json")) as f:
                config = json.load(f)
        m = cls(TivazenConfig.from_json(config, **runtime))
        r = SafetensorsReader(os.path.join(path, "model.safetensors"))
        m.load(r)
        r.close()
        m.finalize()
        return m
