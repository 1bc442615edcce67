"""What every model design of libskainet_cuda's decoder runtime offers to a host (include/skainet_cuda_llama.h): sequence slots,
prompts, single decode steps, logits of chosen positions, greedy generation. The designs (llama.py, tivazen.py, fomalix.py) add how a
model is configured and loaded."""
from __future__ import annotations

import ctypes as C
from typing import Optional, Sequence

import numpy as np

from . import _lib as L


class Decoder:
    """Owner of a model handle. `vocab`, `max_seq` and `max_batch` describe the model behind it."""

    def __init__(self, handle: int, vocab: int, max_seq: int, max_batch: int):
        self.handle = handle
        self.vocab, self.max_seq, self.max_batch = vocab, max_seq, max_batch
        self._free = list(range(max_batch))

    # ---- sequence slots ---------------------------------------------------------------------------
    def acquire(self) -> int:
        """The lowest free sequence slot, emptied."""
        if not self._free:
            raise RuntimeError(f"all {self.max_batch} sequences are in use")
        seq = min(self._free)
        self._free.remove(seq)
        self.reset(seq)
        return seq

    def release(self, seq: int) -> None:
        if seq in self._free or not 0 <= seq < self.max_batch:
            raise ValueError(f"sequence {seq} is not in use")
        self.reset(seq)
        self._free.append(seq)

    def finalize(self) -> None:
        L.check(L.lib().skainet_cuda_llama_finalize(self.handle))

    # ---- running ----------------------------------------------------------------------------------
    def reset(self, seq: Optional[int] = None) -> None:
        """Forgets the tokens of one sequence, or of all."""
        if seq is None:
            L.check(L.lib().skainet_cuda_llama_reset(self.handle))
        else:
            L.check(L.lib().skainet_cuda_llama_reset_seq(self.handle, seq))

    def forward(self, tokens: Sequence[int], want: Sequence[int] = (), seq: int = 0) -> np.ndarray:
        """Runs the next given tokens of a sequence; returns the logits after the places in `want`, [len(want), vocab]."""
        t = np.ascontiguousarray(tokens, dtype=np.int32)
        w = np.ascontiguousarray(want, dtype=np.int32)
        out = np.empty((w.size, self.vocab), dtype=np.float32)
        L.check(L.lib().skainet_cuda_llama_forward(self.handle, seq, t.ctypes.data_as(L.i32p), t.size, w.ctypes.data_as(L.i32p), w.size,
                                                   out.ctypes.data_as(L.f32p)))
        return out

    def prefill(self, tokens: Sequence[int], seq: int = 0, want_next: bool = True) -> Optional[int]:
        t = np.ascontiguousarray(tokens, dtype=np.int32)
        nxt = C.c_int32(-1)
        L.check(L.lib().skainet_cuda_llama_prefill(self.handle, seq, t.ctypes.data_as(L.i32p), t.size, C.byref(nxt) if want_next else None))
        return int(nxt.value) if want_next else None

    def fake_prefill(self, n: int, seq: int = 0, seed: int = 7) -> None:
        L.check(L.lib().skainet_cuda_llama_fake_prefill(self.handle, seq, n, seed))

    def decode(self, tokens_in: np.ndarray, tokens_out: np.ndarray) -> None:
        """One greedy step, host tokens in, host tokens out (int32 arrays of length batch; pinned for best latency)."""
        L.check(L.lib().skainet_cuda_llama_decode(self.handle, tokens_in.size, tokens_in.ctypes.data_as(L.i32p), tokens_out.ctypes.data_as(L.i32p)))

    def decode_ptr(self, batch: int, in_ptr: int, out_ptr: int) -> None:
        L.check(L.lib().skainet_cuda_llama_decode(self.handle, batch, C.cast(in_ptr, L.i32p), C.cast(out_ptr, L.i32p)))

    def generate(self, first_tokens: Sequence[int], n_steps: int) -> np.ndarray:
        """n_steps greedy steps on the device; returns [n_steps, batch] tokens."""
        first = np.ascontiguousarray(first_tokens, dtype=np.int32)
        out = np.empty((n_steps, first.size), dtype=np.int32)
        L.check(L.lib().skainet_cuda_llama_generate(self.handle, first.size, first.ctypes.data_as(L.i32p), n_steps, out.ctypes.data_as(L.i32p)))
        return out

    def logits(self, batch: int = 1) -> np.ndarray:
        out = np.empty((batch, self.vocab), dtype=np.float32)
        L.check(L.lib().skainet_cuda_llama_logits(self.handle, batch, out.ctypes.data_as(L.f32p)))
        return out

    def peek(self, which: int, n: int) -> np.ndarray:
        """Diagnostic read of an activation buffer; what `which` names is the design's (Llama: 0 x, 1 q|k|v, 2 attention out,
        3 gate|up, 4 q; Tivazen: 0 x, 1 merged projection, 16 + j the state X_j of the rows last run; Fomalix: 0 x, 1 merged projection)."""
        out = np.empty(n, dtype=np.float32)
        L.check(L.lib().skainet_cuda_llama_peek(self.handle, which, out.ctypes.data_as(L.f32p), n))
        return out

    def step_cost(self, batch: int = 1) -> tuple[int, int]:
        out = (C.c_int64 * 2)()
        L.check(L.lib().skainet_cuda_llama_step_cost(self.handle, batch, out))
        return int(out[0]), int(out[1])

    @property
    def stream(self) -> int:
        s = C.c_void_p()
        L.check(L.lib().skainet_cuda_llama_stream(self.handle, C.byref(s)))
        return s.value or 0

    def free(self) -> None:
        if self.handle:
            L.lib().skainet_cuda_llama_free(self.handle)
            self.handle = 0

    def __del__(self):
        try:
            self.free()
        except Exception:
            pass
