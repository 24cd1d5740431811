"""Kabidra on the layer-list engine (ugb_hybrid_*, csrc/hybrid_engine.cu)."""
import ctypes as C

import numpy as np

from ._lib import lib
from .device import DType
from .engine import CStruct, EngineModel
from .kabidra_config import LATENT, MINGRU, Config, Layer, weight_names, weight_shapes  # noqa: F401 (re-exported)


class _CConfig(CStruct):
    _fields_ = [(n, C.c_int32) for n in ("width", "vocab", "layers", "conv_taps", "depth_average", "dtype")] + \
               [("eps", C.c_float), ("gain_offset", C.c_float)]


class _CLayer(CStruct):
    _fields_ = [(n, C.c_int32) for n in ("mixer", "width", "heads", "dim", "vdim", "q_rank", "kv_rank")] + \
               [("scale", C.c_float), ("feed_forward", C.c_int32), ("ff", C.c_int32)]


_MIXERS = {MINGRU: 0, LATENT: 1}


class Model(EngineModel):
    """``dtype`` BF16 (serving precision) or F32 (everything in 32 bits)."""

    PREFIX = "ugb_hybrid"

    def __init__(self, cfg, dev, batch, t_max, dtype=DType.BF16):
        self.cfg, self.dev, self.batch, self.dtype = cfg, dev, batch, DType(dtype)
        self.width, self.vocab_local = cfg.width, cfg.vocab
        cc = _CConfig(width=cfg.width, vocab=cfg.vocab, layers=len(cfg.layers), conv_taps=cfg.taps, depth_average=1,
                      dtype=int(self.dtype), eps=cfg.eps, gain_offset=1.0)
        cl = (_CLayer * max(1, len(cfg.layers)))(*[
            _CLayer(mixer=_MIXERS[l.type], feed_forward=int(l.ff is not None), ff=l.ff or 0, **l.mixer) for l in cfg.layers])
        h = C.c_void_p()
        dev._check(lib.ugb_hybrid_create(dev._h, C.byref(cc), C.byref(cl), batch, t_max, C.byref(h)))
        self._h = h

    @classmethod
    def new(cls, cfg, weights, dev, batch, t_max, dtype=DType.BF16):
        """``weights``: name -> host array, uint16 arrays are bf16 bit patterns."""
        m = cls(cfg, dev, batch, t_max, dtype)
        for name, shape in weight_shapes(cfg).items():
            if tuple(weights[name].shape) != shape:
                raise ValueError(f"{name}: shape {tuple(weights[name].shape)}, expected {shape}")
            m.load_weight(name, weights[name])
        return m

    @classmethod
    def from_safetensors(cls, cfg, st, dev, batch, t_max, dtype=DType.BF16):
        m = cls(cfg, dev, batch, t_max, dtype)
        for name, shape in weight_shapes(cfg).items():
            src, got = st.get(name)
            if tuple(got) != shape:
                raise ValueError(f"{name}: shape {tuple(got)}, expected {shape}")
            if src in (DType.BF16, DType.F32):
                _, s = st.load_slice(name, dev)
            else:
                _, s = st.load_slice_with_cast(name, DType.F32, dev)
            m.load_slice(name, s)
        return m

    def layer_outputs(self):
        """f32 [layers, batch, t, width]: the stream after every layer of the last prompt block; set option
        ``keep_layers`` before it."""
        t = self._prefill_t
        out = self._read(4, np.empty((len(self.cfg.layers), self.batch * t, self.width), np.float32))
        return out.reshape(len(self.cfg.layers), self.batch, t, self.width)

    def state_bytes(self, positions):
        """Bytes of state one sequence holds at ``positions`` cached positions."""
        return lib.ugb_hybrid_state_bytes(self._h, positions)

    KERNELS = {"rows": 0, "conv": 1, "gru_in": 2, "gru": 3, "latent_in": 4, "latent_rows": 5, "uq": 6, "absorb": 7,
               "attention": 8, "out": 9, "up": 10, "down": 11, "head": 12, "all": 13}

    def time_kernel(self, name, t=1, iters=20):
        """Milliseconds a decode step (t = 1) or a prompt block of t positions spends in one kind of kernel, all
        layers together, CUDA events around graph replays.  The state is scratch afterwards: reset the model."""
        ms = C.c_float()
        self.dev._check(lib.ugb_hybrid_time_kernel(self._h, self.KERNELS[name], t, iters, C.byref(ms)))
        return ms.value
