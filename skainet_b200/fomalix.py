"""Host-side configuration, loader and handle of the Fomalix design (include/skainet_cuda_fomalix.h): every size and constant
comes from config.json, every tensor from model.safetensors (matrices BF16, [out, in])."""
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

ATTENTION, DELTA, MAMBA2 = 0, 1, 2
W_EMBED, W_HEAD, W_Q, W_K, W_V, W_B, W_A, W_G, W_IN, W_O, W_GATE, W_UP, W_DOWN = range(13)
(V_NORM1, V_NORM1B, V_NORM2, V_NORM2B, V_Q_BIAS, V_K_BIAS, V_V_BIAS, V_SINK, V_Q_CONV, V_K_CONV, V_V_CONV, V_CONV, V_CONV_BIAS, V_A_LOG, V_DT_BIAS, V_D,
 V_MIX_NORM, V_FINAL_NORM) = range(18)


class _Layer(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("type", "heads", "kv_heads", "dim", "vdim", "conv", "norm_groups", "chunk")] + \
               [("scale", C.c_float), ("ff", C.c_int32)]


class _Config(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("n_layers", "width", "vocab")] + [("eps", C.c_float), ("embed_scale", C.c_float)] + \
               [(n, C.c_int32) for n in ("loop_start", "loop_stop", "loop_times", "max_seq", "max_batch", "prefill_rows", "act_f32")]


def _only(d: Dict[str, Any], what: str, *keys: str) -> None:
    extra = sorted(set(d) - set(keys))
    if extra:
        raise ValueError(f"Fomalix: {what} has unknown keys {extra}")


@dataclass
class FomalixLayer:
    type: int
    heads: int
    kv_heads: int                    # query/key heads of the delta rule, groups of Mamba-2
    dim: int                         # query/key size; state size of Mamba-2
    vdim: int
    conv: int = 0
    norm_groups: int = 0
    chunk: int = 0                   # attention: 0 sees every earlier key
    scale: float = 0.0
    ff: int = 0                      # 0: no feed-forward

    @classmethod
    def from_json(cls, d: Dict[str, Any], index: int) -> "FomalixLayer":
        what = f"layer {index}"
        _only(d, what, "type", "mixer", "mlp")
        m = d["mixer"]
        if d["type"] == "attention":
            _only(m, what + " mixer", "heads", "kv_heads", "dim", "vdim", "mask", "scale")
            mask = m.get("mask") or {}
            _only(mask, what + " mask", "size")
            if mask and mask["size"] < 1:
                raise ValueError(f"Fomalix: {what}: chunks of {mask['size']} positions")
            out = cls(ATTENTION, m["heads"], m["kv_heads"], m["dim"], m["vdim"], chunk=mask.get("size", 0), scale=float(m["scale"]))
        elif d["type"] == "delta":
            _only(m, what + " mixer", "heads", "kv_heads", "dim", "vdim", "conv")
            out = cls(DELTA, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"])
        elif d["type"] == "mamba2":
            _only(m, what + " mixer", "heads", "groups", "state", "vdim", "conv", "norm_groups")
            out = cls(MAMBA2, m["heads"], m["groups"], m["state"], m["vdim"], m["conv"], m["norm_groups"])
        else:
            raise ValueError(f"Fomalix: {what}: mixer type {d['type']!r} not supported")
        f = d.get("mlp")
        if f is not None:
            _only(f, what + " mlp", "kind", "ff")
            if f["kind"] != "dense":
                raise ValueError(f"Fomalix: {what}: feed-forward kind {f['kind']!r} not supported")
            out.ff = f["ff"]
        return out

    def to_c(self) -> _Layer:
        return _Layer(self.type, self.heads, self.kv_heads, self.dim, self.vdim, self.conv, self.norm_groups, self.chunk, self.scale, self.ff)


@dataclass
class FomalixConfig:
    width: int
    vocab: int
    eps: float
    layers: List[FomalixLayer]
    embed_scale: float = 1.0
    loop: Optional[tuple] = None     # (start, stop, times)
    max_seq: int = 1024
    max_batch: int = 1
    prefill_rows: int = 0            # rows of one prompt pass, 0: the library's choice
    dtype: str = "bfloat16"          # or "float32": activations, cache and arithmetic in 32-bit

    @classmethod
    def from_json(cls, d: Dict[str, Any], **runtime) -> "FomalixConfig":
        _only(d, "config", "architecture", "embedding", "layers", "loop", "norm", "vocab", "width")
        _only(d["norm"], "norm", "eps")
        _only(d["embedding"], "embedding", "scale")
        loop = d.get("loop")
        if loop is not None:
            _only(loop, "loop", "start", "stop", "times")
            loop = (loop["start"], loop["stop"], loop["times"])
        return cls(d["width"], d["vocab"], float(d["norm"]["eps"]), [FomalixLayer.from_json(l, i) for i, l in enumerate(d["layers"])],
                   float(d["embedding"]["scale"]), loop, **runtime)

    def to_c(self):
        if self.dtype not in ("bfloat16", "float32"):
            raise ValueError(f"Fomalix: dtype {self.dtype!r} is neither bfloat16 nor float32")
        c = _Config(len(self.layers), self.width, self.vocab, self.eps, self.embed_scale, *(self.loop or (0, len(self.layers), 1)), self.max_seq, self.max_batch,
                    self.prefill_rows, int(self.dtype == "float32"))
        return c, (_Layer * len(self.layers))(*[l.to_c() for l in self.layers])


class Fomalix(Decoder):
    architecture = "Fomalix"

    def __init__(self, cfg: FomalixConfig):
        self.cfg = cfg
        h = C.c_int64()
        c, layers = cfg.to_c()
        L.check(L.lib().skainet_cuda_fomalix_create(C.byref(c), layers, C.byref(h)))
        super().__init__(h.value, cfg.vocab, cfg.max_seq, cfg.max_batch)

    # ---- weights --------------------------------------------------------------------------------
    def set_weight(self, layer: int, which: int, w: Weight) -> None:
        """Copies w into the model."""
        L.check(L.lib().skainet_cuda_fomalix_set_weight(self.handle, layer, which, w.handle))

    def set_vector(self, layer: int, which: int, values) -> None:
        v = np.ascontiguousarray(values, dtype=np.float32).reshape(-1)
        L.check(L.lib().skainet_cuda_fomalix_set_vector(self.handle, layer, which, v.ctypes.data_as(L.f32p), v.size))

    def synth(self, seed: int = 100, std: float = 0.02) -> None:
        L.check(L.lib().skainet_cuda_fomalix_synth(self.handle, seed, std))

    def load(self, r: SafetensorsReader) -> None:
        cfg = self.cfg

        def matrix(layer: int, which: int, name: str, rows: int, cols: int) -> None:
            w = r.weight(name, rows, cols)
            self.set_weight(layer, which, w)
            w.free()

        def vector(layer: int, which: int, name: str, *shape: int) -> None:
            v = r.floats(name)
            if v.shape != shape:
                raise ValueError(f"{name}: {list(v.shape)}, expected {list(shape)}")
            self.set_vector(layer, which, v)

        matrix(0, W_EMBED, "embed", cfg.vocab, cfg.width)
        matrix(0, W_HEAD, "head", cfg.vocab, cfg.width)
        vector(0, V_FINAL_NORM, "final.norm", cfg.width)
        for i, l in enumerate(cfg.layers):
            p, W, inner, qk = f"l{i}.", cfg.width, l.heads * l.vdim, l.kv_heads * l.dim
            m = p + "mix."
            vector(i, V_NORM1, p + "norm1", W)
            vector(i, V_NORM1B, p + "norm1b", W)
            if l.type == ATTENTION:
                for w, b, c, n in ((W_Q, V_Q_BIAS, "q", l.heads * l.dim), (W_K, V_K_BIAS, "k", qk), (W_V, V_V_BIAS, "v", l.kv_heads * l.vdim)):
                    matrix(i, w, m + c, n, W)
                    vector(i, b, m + c + ".b", n)
                vector(i, V_SINK, m + "sink", l.heads)
            else:
                vector(i, V_A_LOG, m + "A_log", l.heads)
                vector(i, V_DT_BIAS, m + "dt_bias", l.heads)
            if l.type == DELTA:
                for w, b, c, n in ((W_Q, V_Q_CONV, "q", qk), (W_K, V_K_CONV, "k", qk), (W_V, V_V_CONV, "v", inner)):
                    matrix(i, w, m + c, n, W)
                    vector(i, b, f"{m}{c}.conv", n, l.conv)
                matrix(i, W_B, m + "b", l.heads, W)
                matrix(i, W_A, m + "a", l.heads, W)
                matrix(i, W_G, m + "g", inner, W)
                vector(i, V_MIX_NORM, m + "norm", l.vdim)
            elif l.type == MAMBA2:
                channels = inner + 2 * qk
                matrix(i, W_IN, m + "in", inner + channels + l.heads, W)
                vector(i, V_CONV, m + "conv", channels, l.conv)
                vector(i, V_CONV_BIAS, m + "conv.b", channels)
                vector(i, V_D, m + "D", l.heads)
                vector(i, V_MIX_NORM, m + "norm", inner)
            matrix(i, W_O, m + "o", W, inner)
            if l.ff:
                vector(i, V_NORM2, p + "norm2", W)
                vector(i, V_NORM2B, p + "norm2b", W)
                matrix(i, W_GATE, p + "mlp.gate", l.ff, W)
                matrix(i, W_UP, p + "mlp.up", l.ff, W)
                matrix(i, W_DOWN, p + "mlp.down", W, l.ff)

    @classmethod
    def from_dir(cls, path: str, config: Optional[Dict[str, Any]] = None, **runtime) -> "Fomalix":
        """The model of a folder with config.json and model.safetensors."""
        if config is None:
            with open(os.path.join(path, "config.json")) as f:
                config = json.load(f)
        m = cls(FomalixConfig.from_json(config, **runtime))
        r = SafetensorsReader(os.path.join(path, "model.safetensors"))
        m.load(r)
        r.close()
        m.finalize()
        return m
