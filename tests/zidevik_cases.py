"""Small Zidevik configurations and random weights shared by the Zidevik tests."""
import functools

import numpy as np

from hybrid_cases import logit_err, position_err, write_model  # noqa: F401 (used by the tests)
from oracle import zidevik_ref as Z
from ug_b200 import synth
from ug_b200.zidevik_config import Attention, Config, Experts, Layer, Loop, Scan


def layer(att, scan, mlp, scales=(1.0, 1.0)):
    return Layer(Attention(*att), Scan(*scan), *scales, mlp)


# att: heads, kv_heads, dim, vdim, rotated, base, scale; scan: inner, state, taps, rank.  Sizes that no padding rule divides,
# head widths on both sides of the tensor-core kernels' limits, every feed-forward, loops at either end, and models without a
# loop, a token input or a soft cap.
CONFIGS = {
    "mixed": Config(vocab=211, width=96, eps=1e-5, loop=Loop(1, 3, 2), side_dim=36, logit_softcap=2.0, layers=[
        layer((6, 2, 40, 24, 16, 5000.0, 0.4), (136, 24, 4, 12), 120, (0.8, 1.3)),
        layer((4, 1, 64, 64, 64, 10000.0, 0.3), (72, 8, 3, 8), Experts(5, 2, 56, 72), (1.1, 0.6)),
        layer((3, 3, 24, 48, 8, 300.0, 0.6), (96, 16, 2, 20), None),
        layer((8, 4, 32, 40, 32, 5000.0, 0.5), (40, 33, 4, 5), Experts(8, 1, 40), (1.0, 0.9))]),
    "odd": Config(vocab=101, width=50, eps=3e-4, loop=Loop(0, 2, 3), side_dim=43, logit_softcap=1.5, layers=[
        layer((2, 1, 10, 6, 6, 100.0, 0.9), (35, 5, 2, 3), 33, (0.7, 1.2)),
        layer((3, 1, 14, 9, 14, 700.0, 0.8), (21, 3, 5, 9), Experts(3, 3, 17, 11), (1.4, 0.8))]),
    "wide_heads": Config(vocab=128, width=128, eps=1e-5, loop=Loop(1, 2, 2), side_dim=48, logit_softcap=6.0, layers=[
        layer((4, 2, 128, 128, 96, 10000.0, 0.2), (128, 16, 4, 16), 128),
        layer((34, 2, 72, 56, 72, 2000.0, 0.3), (64, 64, 4, 24), Experts(16, 4, 48, 64), (1.0, 0.5)),
        layer((3, 1, 144, 136, 100, 900.0, 0.25), (200, 100, 3, 40), 64)]),
    "plain": Config(vocab=72, width=80, eps=1e-5, layers=[
        layer((4, 4, 20, 20, 20, 1000.0, 0.5), (80, 16, 1, 8), 96), layer((2, 2, 16, 16, 0, 1.0, 0.7), (48, 12, 4, 4), Experts(4, 2, 32))]),
    "once": Config(vocab=64, width=64, eps=1e-6, loop=Loop(0, 1, 1), side_dim=8, layers=[layer((2, 1, 32, 32, 32, 1.0, 0.4), (64, 8, 4, 8), 64)]),
}


def separate_experts(cfg, w):
    """Sets the choice of experts apart: the first E dimensions of the stream hold a ranking of the experts that depends on
    the token alone and that no sublayer writes to, and the routers read little else.  Rounding never turns a choice round."""
    n = max((l.mlp.count for l in cfg.layers if isinstance(l.mlp, Experts)), default=0)
    if not n:
        return w
    w = {k: synth.bf16_bits_to_f32(v).copy() for k, v in w.items()}
    rng = synth.rng(9)
    for v in range(cfg.vocab):
        w["embed"][v, :n] = 0.4 * rng.permutation(n) - 0.2 * n
    for k, a in w.items():
        tail = k.split(".", 1)[-1]
        if tail.endswith((".o", ".down", "side.proj")):
            a[:n] = 0.0
        elif k == "loop.in":
            a[:n] = 0.0
            a[:n, :n] = np.eye(n)
        elif k == "loop.step":
            a[:, :n] = 0.0
        elif tail == "norm1":
            a[:n] = 1.0
        elif tail == "mlp.router":
            a[:] *= 0.02
            a[:, :len(a)] += 2.0 * np.eye(len(a))
    return {k: synth.to_bf16_bits(a) for k, a in w.items()}


@functools.lru_cache(maxsize=None)
def weights(name, seed=500):
    return separate_experts(CONFIGS[name], synth.zidevik_weights(CONFIGS[name], seed))


def reference(cfg, w):
    return Z.Model(cfg.to_dict(), synth.llama_weights_f32(w))


@functools.lru_cache(maxsize=None)
def oracle(name, seed=500):
    return reference(CONFIGS[name], weights(name, seed))


@functools.lru_cache(maxsize=None)
def oracle_logits(name, tokens, seed=500):
    """float64 [len(tokens), vocab] of one whole sequence (tokens: a tuple)."""
    m = oracle(name, seed)
    return m.fwd(list(tokens), m.new_state())


def tokens(name, seed, n, batch=1):
    return synth.tokens(seed, (batch, n), CONFIGS[name].vocab)


# Largest error of a position, and of the average over the positions compared (eight or more).  A float64 model whose
# activations are rounded to bf16 where the engine stores them reaches 0.066 and 0.011 on these configurations.
LIMITS = {"f32": (2e-5, 1e-5), "bf16": (9e-2, 2.2e-2)}


def agree(got, want, f32, slack=1.0):
    e = position_err(got, want)
    most, mean = LIMITS["f32" if f32 else "bf16"]
    assert np.max(e) < slack * most and (len(e) < 8 or np.mean(e) < slack * mean), (float(np.max(e)), float(np.mean(e)), int(np.argmax(e)))
    return True
