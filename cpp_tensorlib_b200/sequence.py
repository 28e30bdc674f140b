"""Host handle of one sequence on a native decoder: the ``tlb_decoder_*`` surface of
include/tlb200.h that every model shares.  No torch: host buffers are numpy arrays.

The structure follows the reference's captured_decoder and prefill_batched
(bench/cuda/qwen_model.h:357-442, 791-905).
"""
import ctypes as C

import numpy as np

from ._lib import check, lib


class Sequence:
    """A model derives from this, creates its native decoder into ``self.h`` and loads weights."""

    def __init__(self, vocab, max_ctx):
        self.h = C.c_void_p()
        self.vocab, self.max_ctx = vocab, max_ctx
        self.captured = False

    def _stream(self):
        return None

    def set_pos(self, pos):
        check(lib().tlb_decoder_set_pos(self.h, pos, self._stream()))

    def set_token(self, tok):
        check(lib().tlb_decoder_set_token(self.h, int(tok), self._stream()))

    def forward(self):
        check(lib().tlb_decoder_forward(self.h, self._stream()))

    def capture(self):
        check(lib().tlb_decoder_capture(self.h))
        self.captured = True

    def run(self, n):
        check(lib().tlb_decoder_run(self.h, n, self._stream()))

    def step(self, token=None):
        """One token end to end with host buffers: id in, next id out."""
        tin = C.c_int32(-1 if token is None else int(token))
        tout = C.c_int32(0)
        check(lib().tlb_decoder_step(self.h, C.byref(tin), C.byref(tout), self._stream()))
        return int(tout.value)

    def prefill(self, tokens):
        """prefill_batched (bench/cuda/qwen_model.h:423-442): the whole prompt as row-batched
        GEMMs + tiled causal attention from the current position; returns the greedy next
        token, which is also left on the device for run()."""
        ids = (C.c_int32 * len(tokens))(*[int(t) for t in tokens])
        tout = C.c_int32(0)
        check(lib().tlb_decoder_prefill(self.h, ids, len(tokens), C.byref(tout), self._stream()))
        return int(tout.value)

    def host_logits(self):
        """Logits of the last token as a numpy array."""
        out = np.empty(self.vocab, np.float32)
        p = C.c_void_p()
        check(lib().tlb_decoder_logits(self.h, C.byref(p)))
        check(lib().tlb_d2h(out.ctypes.data, p, out.nbytes, self._stream()))
        check(lib().tlb_sync(self._stream()))
        return out

    def extend(self, tokens, want=()):
        """Run the sequence's next tokens -- one by the decode step, more by the prompt pass -- and
        return the logits at the places `want` (increasing) among them, [len(want), vocab]."""
        want = list(want)
        if len(tokens) == 1:
            self.step(tokens[0])
            return self.host_logits()[None] if want else np.empty((0, self.vocab), np.float32)
        ids = np.asarray(tokens, np.int32)
        places = np.asarray(want, np.int32)
        out = np.empty((len(want), self.vocab), np.float32)
        i32p = C.POINTER(C.c_int32)
        tout = C.c_int32(0)
        check(lib().tlb_decoder_prefill_logits(self.h, ids.ctypes.data_as(i32p), len(ids), places.ctypes.data_as(i32p),
                                               len(want), out.ctypes.data, C.byref(tout), self._stream()))
        return out

    def generate(self, prompt, n):
        """`n` greedy tokens behind `prompt`, from the start of a new sequence."""
        if not self.captured:
            self.capture()
        self.set_pos(0)
        out = [self.prefill(prompt) if len(prompt) > 1 else self.step(prompt[0])]
        while len(out) < n:
            out.append(self.step())
        return out[:n]

    def last_token(self):
        t = C.c_int32(0)
        check(lib().tlb_decoder_last_token(self.h, C.byref(t), self._stream()))
        return int(t.value)

    def launches_per_token(self):
        return int(lib().tlb_decoder_launches_per_token(self.h))

    def close(self):
        if self.h:
            check(lib().tlb_decoder_destroy(self.h))
            self.h = None
