"""Comparisons and buffers shared by the tests of the models on the layer-list engine."""
import json
import struct

import numpy as np

from ug_b200 import synth


class Buf:
    """Host arrays in the activation type of a test: f32, or f32 values that bf16 holds exactly."""

    def __init__(self, dev, bf16):
        self.dev, self.bf16 = dev, bf16

    def act(self, x):
        """(device slice, the values it holds as float64)"""
        x = np.ascontiguousarray(x, np.float32)
        if not self.bf16:
            return self.dev.slice_from_values(x.ravel()), x.astype(np.float64)
        bits = synth.to_bf16_bits(x)
        return self.dev.slice_from_values(bits.ravel(), bf16=True), synth.bf16_bits_to_f32(bits).astype(np.float64)

    def f32(self, x):
        return self.dev.slice_from_values(np.ascontiguousarray(x, np.float32).ravel())

    def out(self, n):
        from ug_b200 import DType
        return self.dev.allocate_uninit(DType.BF16 if self.bf16 else DType.F32, n)

    def read(self, s, shape):
        v = s.to_vec()
        return (synth.bf16_bits_to_f32(v) if v.dtype == np.uint16 else v).reshape(shape).astype(np.float64)

    @property
    def tol(self):
        return 8e-3 if self.bf16 else 2e-5


def close(got, want, tol):
    return float(np.max(np.abs(got - want)) / max(np.max(np.abs(want)), 1e-30)) < tol


def position_err(got, want):
    """Per position: rms(difference without its mean) / rms(all oracle logits without their mean)."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    w = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt(np.mean(d * d, axis=-1)) / np.sqrt(np.mean(w * w))


def logit_err(got, want):
    return float(np.max(position_err(got, want)))


# Largest error of a position, and of the average over the positions compared.  bf16 rounding is amplified most where
# two keys or the two sides of a branch are close, hence the distance between the two limits.
LIMITS = {"f32": (2e-5, 1e-5), "bf16": (6e-2, 2.5e-2)}


def agree(got, want, f32, slack=1.0):
    e = position_err(got, want)
    most, mean = LIMITS["f32" if f32 else "bf16"]
    assert np.max(e) < slack * most and np.mean(e) < slack * mean, (float(np.max(e)), float(np.mean(e)), int(np.argmax(e)))
    return True


def write_model(folder, cfg, w):
    """config.json and model.safetensors (uint16 arrays as BF16)."""
    (folder / "config.json").write_text(json.dumps(cfg.to_dict()))
    header, blobs, at = {}, [], 0
    for name, a in w.items():
        raw = np.ascontiguousarray(a).tobytes()
        header[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    h = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(h)) + h + b"".join(blobs))
