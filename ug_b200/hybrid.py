"""Models on the layer-list engine (ugb_hybrid_*, csrc/hybrid_engine.cu): a subclass turns its configuration into the
engine's descriptors and lists its tensors."""
import ctypes as C

import numpy as np

from ._lib import lib
from .device import DType
from .engine import CStruct, EngineModel

FORM_SANDWICH, FORM_PARALLEL = 0, 1
MIXER_MINGRU, MIXER_LATENT_ATTENTION, MIXER_ATTENTION_SCAN = 0, 1, 2
FF_NONE, FF_RELU2, FF_GATED, FF_EXPERTS = 0, 1, 2, 3


class CConfig(CStruct):
    _fields_ = [(n, C.c_int32) for n in ("width", "vocab", "layers", "conv_taps", "depth_average", "dtype")] + \
               [("eps", C.c_float), ("gain_offset", C.c_float)] + \
               [(n, C.c_int32) for n in ("form", "loop_start", "loop_stop", "loop_times", "side_dim")] + [("logit_softcap", C.c_float)]


class CLayer(CStruct):
    _fields_ = [(n, C.c_int32) for n in ("mixer", "width", "heads", "dim", "vdim", "q_rank", "kv_rank")] + \
               [("scale", C.c_float), ("feed_forward", C.c_int32), ("ff", C.c_int32)] + \
               [(n, C.c_int32) for n in ("kv_heads", "rot_dims", "rot_interleaved", "qk_norm")] + \
               [("rot_base", C.c_float), ("attention_scale", C.c_float)] + \
               [(n, C.c_int32) for n in ("inner", "state", "conv", "dt_rank")] + [("scan_scale", C.c_float)] + \
               [(n, C.c_int32) for n in ("experts", "top", "expert_ff")]


class HybridModel(EngineModel):
    """``dtype`` BF16 (serving precision) or F32 (everything in 32 bits)."""

    PREFIX = "ugb_hybrid"
    layer_runs = 0               # passes over layers of one step

    def __init__(self, cfg, dev, batch, t_max, dtype=DType.BF16):
        self.cfg, self.dev, self.batch, self.dtype = cfg, dev, batch, DType(dtype)
        self.width, self.vocab_local = cfg.width, cfg.vocab
        cc, layers = self.describe(cfg)
        cc.width, cc.vocab, cc.layers, cc.dtype, cc.eps = cfg.width, cfg.vocab, len(layers), int(self.dtype), cfg.eps
        self.layer_runs = len(layers) + max(0, cc.loop_times - 1) * (cc.loop_stop - cc.loop_start)
        cl = (CLayer * max(1, len(layers)))(*layers)
        h = C.c_void_p()
        dev._check(lib.ugb_hybrid_create(dev._h, C.byref(cc), C.byref(cl), batch, t_max, C.byref(h)))
        self._h = h

    @staticmethod
    def describe(cfg):
        """(CConfig, [CLayer]): everything but width, vocabulary, layer count, precision and eps."""
        raise NotImplementedError

    @staticmethod
    def weight_shapes(cfg):
        """Tensor name -> shape, in load order."""
        raise NotImplementedError

    @classmethod
    def new(cls, cfg, weights, dev, batch, t_max, dtype=DType.BF16):
        """``weights``: name -> host array, uint16 arrays are bf16 bit patterns."""
        m = cls(cfg, dev, batch, t_max, dtype)
        for name, shape in cls.weight_shapes(cfg).items():
            if tuple(weights[name].shape) != shape:
                raise ValueError(f"{name}: shape {tuple(weights[name].shape)}, expected {shape}")
            m.load_weight(name, weights[name])
        return m

    @classmethod
    def from_safetensors(cls, cfg, st, dev, batch, t_max, dtype=DType.BF16):
        m = cls(cfg, dev, batch, t_max, dtype)
        for name, shape in cls.weight_shapes(cfg).items():
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
        """f32 [layer runs, batch, t, width]: the stream after every layer run of the last prompt block; set option
        ``keep_layers`` before it."""
        t = self._prefill_t
        out = self._read(4, np.empty((self.layer_runs, self.batch * t, self.width), np.float32))
        return out.reshape(self.layer_runs, self.batch, t, self.width)

    def state_bytes(self, positions):
        """Bytes of state one sequence holds at ``positions`` cached positions."""
        return lib.ugb_hybrid_state_bytes(self._h, positions)

    KERNELS = {"rows": 0, "conv": 1, "gru_in": 2, "gru": 3, "latent_in": 4, "latent_rows": 5, "uq": 6, "absorb": 7,
               "attention": 8, "out": 9, "up": 10, "down": 11, "head": 12, "mix_in": 13, "mix_rows": 14, "scan_in": 15,
               "scan": 16, "route": 17, "expert_up": 18, "expert_down": 19, "side": 20, "side_gate": 21, "loop": 22, "all": 23}

    def time_kernel(self, name, t=1, iters=20):
        """Milliseconds a decode step (t = 1) or a prompt block of t positions spends in one kind of kernel, all
        layers together, CUDA events around graph replays.  The state is scratch afterwards: reset the model."""
        ms = C.c_float()
        self.dev._check(lib.ugb_hybrid_time_kernel(self._h, self.KERNELS[name], t, iters, C.byref(ms)))
        return ms.value
