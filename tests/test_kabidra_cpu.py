"""CPU checks of the Kabidra oracle and of the pure-Python side of the model: the oracle against closed forms, its
continuation from any cut, the sensitivity of the test models to every mechanism, configuration and registry."""
import json

import numpy as np
import pytest

from kabidra_cases import CONFIGS, logit_err, oracle, oracle_logits, tokens, weights
from oracle import kabidra_ref as K
from ug_b200 import kabidra_config as KC
from ug_b200 import synth


def test_norms_and_candidate():
    x = synth.normal(1, (5, 33)).astype(np.float64)
    w = synth.normal(2, (33,)).astype(np.float64)
    ref = x / np.sqrt((x ** 2).sum(-1, keepdims=True) / 33 + 1e-3)
    assert np.allclose(K.norm_plain(x, w, 1e-3), ref * w)
    assert np.allclose(K.norm_centred(x, w, 1e-3), ref + ref * w)
    u = np.array([-30.0, -1e-9, 0.0, 1e-9, 4.0])
    assert np.allclose(K.gru_candidate(u), [0.0, 0.5, 0.5, 0.5, 4.5], atol=1e-8)
    assert np.array_equal(K.relu_squared(np.array([-2.0, 0.0, 3.0])), [0.0, 0.0, 9.0])


def test_causal_conv_is_a_shifted_sum():
    h, w = synth.normal(3, (9, 4)).astype(np.float64), synth.normal(4, (4, 3)).astype(np.float64)
    out, tail = K.causal_conv(h, w, np.zeros((2, 4)))
    want = w[:, 2] * h
    want[1:] += w[:, 1] * h[:-1]
    want[2:] += w[:, 0] * h[:-2]
    assert np.allclose(out, want) and np.array_equal(tail, h[-2:])


def test_min_gru_closed_form():
    z, c = K.sigmoid(synth.normal(5, (12, 3))), synth.normal(6, (12, 3)).astype(np.float64)
    s, last = K.min_gru(z, c, np.full(3, 2.0))
    keep = np.prod(1 - z, axis=0)
    want = keep * 2.0 + sum(z[j] * c[j] * np.prod(1 - z[j + 1:], axis=0) for j in range(12))
    assert np.allclose(last, want) and np.allclose(s[-1], last)


def test_latent_attention_equals_its_absorbed_form():
    rng = np.random.default_rng(7)
    q, c = rng.standard_normal((4, 3, 5)), rng.standard_normal((10, 8))
    uk, uv = rng.standard_normal((15, 8)), rng.standard_normal((18, 8))
    out = K.latent_attention(q, c, uk, uv, 0.4, 6, 3)
    for i in range(4):
        for h in range(3):
            p = K.softmax(c[:7 + i] @ (uk[5 * h:5 * h + 5].T @ q[i, h]) * 0.4)
            assert np.allclose(out[i, h], uv[6 * h:6 * h + 6] @ (p @ c[:7 + i]))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_oracle_continues_from_any_cut(name):
    m, toks = oracle(name), [int(x) for x in tokens(name, 8, 23)[0]]
    whole = oracle_logits(name, tuple(toks))
    st, got, at = m.new_state(), [], 0
    for n in (1, 2, 7, 1, 1, 8, 3):
        got.append(m.fwd(toks[at:at + n], st))
        at += n
    assert at == 23 and np.max(np.abs(np.concatenate(got) - whole)) < 1e-9


class _Without(K.Model):
    """The oracle with one mechanism left out: what the test models have to be able to tell apart."""

    def __init__(self, name, what):
        super().__init__(CONFIGS[name].to_dict(), synth.llama_weights_f32(weights(name)))
        w = self.w
        for k in list(w):
            tail = k.split(".", 1)[-1]
            if what == "bias" and tail.endswith(".b"):
                w[k] = np.zeros_like(w[k])
            if what == "oldest tap" and tail.startswith("canon"):
                w[k] = w[k].copy()
                w[k][:, 0] = 0.0
            if what == "depth average" and tail == "dwa":
                w[k] = np.eye(len(w[k]))[-1]
            if what == "norm gain" and tail in ("norm1", "norm1b", "norm2", "norm2b", "embed.norm", "final.norm", "norm"):
                w[k] = np.zeros_like(w[k])
            if what == "head gate" and tail == "mix.g" and "l%s.mix.dq" % k[1:k.index(".")] in w:
                w[k] = np.zeros_like(w[k])


@pytest.mark.parametrize("name,what", [("mixed", w) for w in ("bias", "oldest tap", "depth average", "norm gain", "head gate")] +
                         [("odd", w) for w in ("bias", "oldest tap", "depth average", "head gate")])
def test_models_show_a_missing_mechanism(name, what):
    """A mechanism left out moves the logits by more than the GPU tests allow in bf16, let alone in f32."""
    toks = tuple(int(x) for x in tokens(name, 9, 20)[0])
    m = _Without(name, what)
    assert logit_err(m.fwd(list(toks), m.new_state()), oracle_logits(name, toks)) > 0.1


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_models_show_a_lost_state(name):
    """A sequence whose state is dropped at a cut, or that sees the state of another one, is told apart at once."""
    toks = [int(x) for x in tokens(name, 10, 24)[0]]
    want = oracle_logits(name, tuple(toks))
    m = oracle(name)
    for key in ("canon1", "canon2", "s", "c"):
        st = m.new_state()
        m.fwd(toks[:16], st)
        fresh = m.new_state()
        for a, b in zip(st["layers"], fresh["layers"]):
            if key in a:
                a[key] = b[key] if key != "c" else a[key] * 0.0
        got = m.fwd(toks[16:17], st)
        assert logit_err(got, want[16:17]) > 0.1, key


def test_config_round_trip_and_shapes():
    for cfg in CONFIGS.values():
        again = KC.Config.from_dict(json.loads(json.dumps(cfg.to_dict())))
        assert again == cfg
        shapes = KC.weight_shapes(cfg)
        assert list(shapes) == KC.weight_names(cfg)
        assert shapes[f"l{len(cfg.layers) - 1}.dwa"] == (len(cfg.layers) + 1,)
        for i, l in enumerate(cfg.layers):
            assert (f"l{i}.mlp.up" in shapes) == (l.ff is not None) == (f"l{i}.canon2" in shapes)
    bad = CONFIGS["mixed"].to_dict()
    bad["layers"][0]["type"] = "something"
    with pytest.raises(ValueError):
        KC.Config.from_dict(bad)


def test_registry_names_architectures(tmp_path):
    from ug_b200 import UgError, registry
    assert registry.architecture(CONFIGS["odd"].to_dict()) == "Kabidra"
    assert registry.architecture({"architectures": ["LlamaForCausalLM"]}) == "Llama"
    assert registry.architecture({"hidden_size": 8, "num_key_value_heads": 1}) == "Llama"
    for bad in ({"architecture": "Unknown"}, {"model_type": "other"}, {}):
        with pytest.raises(UgError):
            registry.architecture(bad)
    with pytest.raises(UgError):
        registry.weight_files(str(tmp_path))
