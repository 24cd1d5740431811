"""Host side of the fused decoder engines: what every model of this package does with its engine handle.

A subclass names its entry points (``PREFIX``: ugb_<engine>_decode, _prefill, _read, ...) and creates the handle;
steps, prompts, reads and weight upload are the same for all of them.
"""
import ctypes as C

import numpy as np

from ._lib import lib
from .device import UgError


class EngineModel:
    """``batch`` independent sequences at one shared position, greedy choice on the device."""

    PREFIX = None
    READ_LOGITS, READ_NEXT, READ_HIDDEN, READ_PREFILL_LOGITS = 0, 1, 2, 3

    dev = None
    _h = None
    batch = 0
    vocab_local = 0        # logit columns this process holds
    width = 0              # of the residual stream

    def _fn(self, name):
        return getattr(lib, f"{self.PREFIX}_{name}")

    def _read(self, what, out):
        self.dev._check(self._fn("read")(self._h, what, out.ctypes.data, out.size))
        return out

    def load_weight(self, name, arr):
        """One tensor by its safetensors name; uint16 arrays are bf16 bit patterns."""
        arr = np.ascontiguousarray(arr)
        self.load_slice(name, self.dev.slice_from_values(arr.ravel(), bf16=(arr.dtype == np.uint16)))

    def load_slice(self, name, s):
        self.dev._check(self._fn("load_weight")(self._h, name.encode(), s._h))
        self.dev.synchronize()

    def close(self):
        h, self._h = self._h, None
        if h:
            self._fn("destroy")(h)

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass

    def set_option(self, key, value):
        self.dev._check(self._fn("set_option")(self._h, key.encode(), value))

    def reset(self, pos=0):
        self.dev._check(self._fn("reset")(self._h, pos))

    @property
    def position(self):
        return self._fn("position")(self._h)

    def fwd(self, tokens):
        """Model::fwd on explicit token ids, asynchronous: int32 [batch] or [batch, 1] is one
        decode step; [batch, t] with t > 1 appends t positions (causal prefill) and keeps the
        logits of every position for :meth:`prefill_logits`."""
        tokens = np.ascontiguousarray(tokens, dtype=np.int32)
        if tokens.ndim == 2 and tokens.shape[1] > 1:
            return self.prefill(tokens, all_logits=True)
        s = self.dev.slice_from_values(tokens.reshape(-1))
        self.dev._check(self._fn("decode")(self._h, s._h, 1))

    def prefill(self, tokens, all_logits=False):
        """Appends ``tokens`` (int32 [batch, t], host array or device Slice of batch*t ids) to
        every sequence; :meth:`logits` / :meth:`next_tokens` then refer to the last position."""
        if isinstance(tokens, np.ndarray) or not hasattr(tokens, "_h"):
            tokens = np.ascontiguousarray(tokens, dtype=np.int32)
            if tokens.ndim != 2 or tokens.shape[0] != self.batch:
                raise UgError(4, f"prefill tokens must be [batch={self.batch}, t], got {tokens.shape}")
            t = tokens.shape[1]
            s = self.dev.slice_from_values(tokens.reshape(-1))
        else:
            s, t = tokens, tokens.len // self.batch
        self.dev._check(self._fn("prefill")(self._h, s._h, t, int(all_logits)))
        self._prefill_t = t if all_logits else getattr(self, "_prefill_t", 0)

    def prefill_logits(self):
        """f32 [batch, t, vocab] of the last ``all_logits`` prefill (what Model::fwd returns)."""
        t = getattr(self, "_prefill_t", 0)
        return self._read(self.READ_PREFILL_LOGITS, np.empty((self.batch, t, self.vocab_local), np.float32))

    def decode(self, n_steps):
        """Greedy decoding: each step feeds the previous step's argmax; asynchronous."""
        self.dev._check(self._fn("decode")(self._h, None, n_steps))

    def logits(self):
        """f32 [batch, vocab]; a tensor-parallel rank returns its columns
        [vocab_offset, vocab_offset + vocab_local)."""
        return self._read(self.READ_LOGITS, np.empty((self.batch, self.vocab_local), np.float32))

    def next_tokens(self):
        return self._read(self.READ_NEXT, np.empty(self.batch, np.int32))

    def hidden(self):
        return self._read(self.READ_HIDDEN, np.empty((self.batch, self.width), np.float32))


class CStruct(C.Structure):
    """ctypes structure built from keyword arguments; unnamed fields are zero."""

    def __init__(self, **kw):
        super().__init__()
        known = {f[0] for f in self._fields_}
        for k, v in kw.items():
            if k not in known:
                raise TypeError(f"{type(self).__name__} has no field {k}")
            setattr(self, k, v)
