"""Small Kabidra configurations, random weights and comparisons shared by the Kabidra tests."""
import functools
import json
import struct

import numpy as np

from oracle import kabidra_ref as K
from ug_b200 import synth
from ug_b200.kabidra_config import LATENT, MINGRU, Config, Layer


def att(heads, dim, vdim, q_rank, kv_rank, scale, ff):
    return Layer(LATENT, dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale), ff)


def gru(width, ff):
    return Layer(MINGRU, dict(width=width), ff)


# Sizes that no padding rule divides, sizes that coincide, layers with and without a feed-forward, head widths on both
# sides of the tensor-core kernels' limits.  A scale well above 1 / sqrt(dim) makes the softmax pick single keys.
CONFIGS = {
    "mixed": Config(vocab=211, width=96, eps=1e-5, taps=4,
                    layers=[gru(136, 160), att(3, 24, 40, 56, 72, 0.6, 88), gru(96, None), att(5, 64, 64, 32, 128, 0.4, None), gru(40, 72)]),
    "odd": Config(vocab=101, width=50, eps=3e-4, taps=2,
                  layers=[att(1, 10, 6, 7, 9, 1.1, 33), gru(35, 21), att(2, 7, 12, 20, 13, 0.9, 50)]),
    "one_tap": Config(vocab=64, width=64, eps=1e-6, taps=1, layers=[gru(64, 64), gru(64, 64)]),
    "wide_heads": Config(vocab=128, width=128, eps=1e-5, taps=7,
                         layers=[att(2, 128, 128, 96, 256, 0.2, 128), att(17, 48, 72, 64, 100, 0.5, 96), gru(200, 64)]),
    "wider_heads": Config(vocab=96, width=72, eps=1e-5, taps=3,
                          layers=[att(2, 144, 136, 40, 80, 0.25, 64), gru(72, 40), att(3, 32, 200, 40, 56, 0.5, None)]),
    "long_latent": Config(vocab=80, width=64, eps=1e-5, taps=3, layers=[att(4, 32, 32, 48, 560, 0.5, 64), gru(48, 64)]),
    "attention_only": Config(vocab=72, width=80, eps=1e-5, taps=5, layers=[att(4, 20, 20, 24, 300, 0.7, None)]),
}


@functools.lru_cache(maxsize=None)
def weights(name, seed=300):
    return synth.kabidra_weights(CONFIGS[name], seed)


@functools.lru_cache(maxsize=None)
def oracle(name, seed=300):
    return K.Model(CONFIGS[name].to_dict(), synth.llama_weights_f32(weights(name, seed)))


@functools.lru_cache(maxsize=None)
def oracle_logits(name, tokens, seed=300):
    """float64 [len(tokens), vocab] of one whole sequence (tokens: a tuple)."""
    m = oracle(name, seed)
    return m.fwd(list(tokens), m.new_state())


def tokens(name, seed, n, batch=1):
    return synth.tokens(seed, (batch, n), CONFIGS[name].vocab)


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
