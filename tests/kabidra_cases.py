"""Small Kabidra configurations, random weights and comparisons shared by the Kabidra tests."""
import functools

from hybrid_cases import agree, logit_err, position_err, write_model  # noqa: F401 (used by the tests)
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
