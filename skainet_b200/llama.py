"""Host-side handle of the Llama-style design of the decoder runtime inside libskainet_cuda (include/skainet_cuda_llama.h)."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import numpy as np

from . import _lib as L
from .decoder import Decoder
from .device import Weight

W_EMBED, W_HEAD, W_OUT_NORM, W_ATTN_NORM, W_Q, W_K, W_V, W_O, W_FFN_NORM, W_GATE, W_UP, W_DOWN, W_QKV, W_GATE_UP = range(14)


class _Config(C.Structure):
    _fields_ = [(n, C.c_int32) for n in ("n_layers", "d_model", "n_heads", "n_kv_heads", "head_dim", "ffn_dim", "vocab")] + \
               [("rms_eps", C.c_float), ("rope_theta", C.c_float)] + \
               [(n, C.c_int32) for n in ("rope_mode", "max_seq", "max_batch", "linear_enc", "table_enc", "tp_rank", "tp_world")]


@dataclass
class LlamaConfig:
    n_layers: int
    d_model: int
    n_heads: int
    n_kv_heads: int
    head_dim: int
    ffn_dim: int
    vocab: int
    rms_eps: float = 1e-5
    rope_theta: float = 1e4
    rope_mode: int = 0
    max_seq: int = 1024
    max_batch: int = 1
    linear_enc: str = "Q4_K"
    table_enc: str = "Q8_0"
    tp_rank: int = 0
    tp_world: int = 1

    @classmethod
    def llama7b(cls, **kw) -> "LlamaConfig":
        """Llama-7B shape: 32 layers, d 4096, FFN 11008, 32 heads, vocab 32000; Q4_K linears, Q8_0 embed/output."""
        return cls(32, 4096, 32, 32, 128, 11008, 32000, **kw)

    @classmethod
    def llama70b(cls, **kw) -> "LlamaConfig":
        """Llama-70B-class shape: 80 layers, d 8192, FFN 28672, 64 q / 8 kv heads, vocab 128256, all Q4_K."""
        kw.setdefault("table_enc", "Q4_K")
        return cls(80, 8192, 64, 8, 128, 28672, 128256, **kw)

    def to_c(self) -> _Config:
        return _Config(self.n_layers, self.d_model, self.n_heads, self.n_kv_heads, self.head_dim, self.ffn_dim, self.vocab,
                       self.rms_eps, self.rope_theta, self.rope_mode, self.max_seq, self.max_batch, L.ENC[self.linear_enc],
                       L.ENC[self.table_enc], self.tp_rank, self.tp_world)


class Llama(Decoder):
    def __init__(self, cfg: LlamaConfig):
        self.cfg = cfg
        h = C.c_int64()
        c = cfg.to_c()
        L.check(L.lib().skainet_cuda_llama_create(C.byref(c), C.byref(h)))
        super().__init__(h.value, cfg.vocab, cfg.max_seq, cfg.max_batch)

    @classmethod
    def from_gguf(cls, path: str, max_seq: int = 1024, max_batch: int = 1) -> "Llama":
        """The model of a GGUF file of architecture "llama" (the file's own tensor names and metadata keys)."""
        from .gguf import StreamingGGUFReader
        r = StreamingGGUFReader(path)
        f = lambda key, default=None: r.fields.get("llama." + key, default)
        vocab, d_model = r.tensor("token_embd.weight").shape
        heads = f("attention.head_count")
        cfg = LlamaConfig(f("block_count"), d_model, heads, f("attention.head_count_kv", heads), f("attention.key_length", d_model // heads),
                          f("feed_forward_length"), vocab, rms_eps=f("attention.layer_norm_rms_epsilon", 1e-5), rope_theta=f("rope.freq_base", 1e4),
                          max_seq=max_seq, max_batch=max_batch, linear_enc=r.tensor("blk.0.attn_q.weight").encoding,
                          table_enc=r.tensor("token_embd.weight").encoding)
        m = cls(cfg)
        names = {t.name for t in r.tensors}
        m.set_weight(0, W_EMBED, r.loadWeightToDevice("token_embd.weight"))
        m.set_weight(0, W_HEAD, r.loadWeightToDevice("output.weight" if "output.weight" in names else "token_embd.weight"))
        m.set_norm(0, W_OUT_NORM, r.loadFloats("output_norm.weight"))
        for l in range(cfg.n_layers):
            for which, name in ((W_Q, "attn_q"), (W_K, "attn_k"), (W_V, "attn_v"), (W_O, "attn_output"), (W_GATE, "ffn_gate"), (W_UP, "ffn_up"), (W_DOWN, "ffn_down")):
                m.set_weight(l, which, r.loadWeightToDevice(f"blk.{l}.{name}.weight"))
            for which, name in ((W_ATTN_NORM, "attn_norm"), (W_FFN_NORM, "ffn_norm")):
                m.set_norm(l, which, r.loadFloats(f"blk.{l}.{name}.weight"))
        r.close()
        m.finalize()
        return m

    # ---- weights --------------------------------------------------------------------------------
    def set_weight(self, layer: int, which: int, w: Weight) -> None:
        L.check(L.lib().skainet_cuda_llama_set_weight(self.handle, layer, which, w.handle))
        w.handle = 0      # the model owns it now

    def set_norm(self, layer: int, which: int, gamma: np.ndarray) -> None:
        g = np.ascontiguousarray(gamma, dtype=np.float32)
        assert g.size == self.cfg.d_model
        L.check(L.lib().skainet_cuda_llama_set_norm(self.handle, layer, which, g.ctypes.data_as(L.f32p)))

    def synth(self, seed: int = 100, std: float = 0.02) -> None:
        L.check(L.lib().skainet_cuda_llama_synth(self.handle, seed, std))

    def export_weight(self, layer: int, which: int) -> np.ndarray:
        """Canonical row-major packed bytes of this rank's shard of a tensor."""
        h = C.c_int64()
        L.check(L.lib().skainet_cuda_llama_get_weight(self.handle, layer, which, C.byref(h)))
        info = (C.c_int64 * 4)()
        L.check(L.lib().skainet_cuda_weight_info(h.value, info))
        out = np.empty(int(info[3]), dtype=np.uint8)
        L.check(L.lib().skainet_cuda_weight_export(h.value, out.ctypes.data_as(L.u8p), out.size))
        return out

    def weight(self, layer: int, which: int) -> Weight:
        """A borrowed view of a tensor the model owns (do not free)."""
        h = C.c_int64()
        L.check(L.lib().skainet_cuda_llama_get_weight(self.handle, layer, which, C.byref(h)))
        w = Weight(h.value)
        w.free = lambda: None      # borrowed
        return w

    @staticmethod
    def tp_unique_id() -> bytes:
        buf = (C.c_uint8 * 128)()
        L.check(L.lib().skainet_cuda_llama_tp_unique_id(buf))
        return bytes(buf)

    def tp_init(self, unique_id: bytes) -> None:
        buf = (C.c_uint8 * 128).from_buffer_copy(unique_id)
        L.check(L.lib().skainet_cuda_llama_tp_init(self.handle, buf))

    def tp_exchange_time(self, mode: int, rounds: int = 64, reps: int = 20) -> float:
        """Device microseconds of one group exchange of a [d_model] row, timed on its own (collective: all ranks call it).
        mode 0 peer-memory sum, 1 store + gather + sum + RMSNorm + quantize, 2 NCCL sum."""
        out = C.c_float()
        L.check(L.lib().skainet_cuda_llama_tp_exchange_time(self.handle, mode, rounds, reps, C.byref(out)))
        return float(out.value)
