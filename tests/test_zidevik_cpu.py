"""CPU checks of the Zidevik oracle and of the pure-Python side of the model: the oracle against closed forms, its
continuation from any cut, the sensitivity of the test models to every mechanism, configuration and registry."""
import json

import numpy as np
import pytest

from oracle import zidevik_ref as Z
from ug_b200 import synth
from ug_b200 import zidevik_config as ZC
from zidevik_cases import CONFIGS, logit_err, oracle, oracle_logits, tokens, weights


def test_rotation_keeps_lengths_and_relative_angles():
    x = synth.normal(1, (6, 2, 12)).astype(np.float64)
    r = Z.rotate(x, np.arange(6), 50.0, 8)
    assert np.allclose(np.linalg.norm(r[..., :8], axis=-1), np.linalg.norm(x[..., :8], axis=-1))
    assert np.array_equal(r[..., 8:], x[..., 8:]) and np.array_equal(r[0], x[0])
    a, b = x[:1], x[1:2]
    dot = lambda p, q: float(np.sum(Z.rotate(a, [p], 50.0, 8) * Z.rotate(b, [q], 50.0, 8)))
    assert abs(dot(3, 10) - dot(103, 110)) < 1e-9 and abs(dot(3, 10) - dot(3, 11)) > 1e-3
    one = np.zeros((1, 1, 4))
    one[0, 0, 2] = 1.0
    assert np.allclose(Z.rotate(one, [7], 9.0, 4)[0, 0], [0, 0, np.cos(7 / 3), np.sin(7 / 3)])


def test_attention_shares_key_heads():
    rng = np.random.default_rng(2)
    q, k, v = rng.standard_normal((3, 6, 5)), rng.standard_normal((7, 2, 5)), rng.standard_normal((7, 2, 4))
    out = Z.grouped_attention(q, k, v, 0.7, 4)
    for i in range(3):
        for h in range(6):
            p = np.exp(k[:5 + i, h // 3] @ q[i, h] * 0.7)
            assert np.allclose(out[i, h], (p / p.sum()) @ v[:5 + i, h // 3])


def test_convolution_is_a_shifted_sum():
    h, w, b = (synth.normal(s, n).astype(np.float64) for s, n in ((3, (9, 4)), (4, (4, 3)), (5, (4,))))
    out, tail = Z.causal_conv(h, w, b, np.zeros((2, 4)))
    want = w[:, 2] * h + b
    want[1:] += w[:, 1] * h[:-1]
    want[2:] += w[:, 0] * h[:-2]
    assert np.allclose(out, Z.silu(want)) and np.array_equal(tail, h[-2:])


def test_scan_closed_form():
    t, n, s = 11, 3, 4
    x, dt, a = synth.normal(5, (t, n)), Z.softplus(synth.normal(6, (t, n))), -np.exp(synth.normal(7, (n, s)))
    b, c, d, s0 = synth.normal(8, (t, s)), synth.normal(9, (t, s)), synth.normal(10, (n,)), synth.normal(11, (n, s))
    y, last = Z.selective_scan(x, dt, a, b, c, d, s0)
    for i in range(t):
        age = lambda j: np.exp(dt[j + 1:i + 1].sum(0)[:, None] * a)
        state = np.exp(dt[:i + 1].sum(0)[:, None] * a) * s0 + sum(age(j) * (dt[j] * x[j])[:, None] * b[j] for j in range(i + 1))
        assert np.allclose(y[i], state @ c[i] + d * x[i])
    assert np.allclose(last, state)


def test_small_functions():
    z = np.array([0.3, -2.0, 5.0, 5.0, 1.0])
    e, s = Z.route(z, 3)
    assert list(e) == [2, 3, 4] and np.allclose(s, 1 / (1 + np.exp(-z[e])))
    x = np.array([-60.0, -1.0, 0.0, 2.0, 60.0])
    assert np.allclose(Z.softplus(x), [0.0, np.log1p(np.exp(-1)), np.log(2), np.log1p(np.exp(2)), 60.0])
    assert np.allclose(Z.gelu_tanh(x), [0.0, -0.158808, 0.0, 1.954598, 60.0], atol=1e-6)
    assert np.allclose(Z.softcap(x, 3.0), 3 * np.tanh(x / 3)) and np.array_equal(Z.softcap(x, None), x)


def test_layer_runs():
    cfg = {"layers": [None] * 5, "loop": {"start": 1, "stop": 3, "times": 2}}
    assert Z.layer_runs(cfg) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None), (4, None)]
    assert Z.layer_runs({"layers": [None] * 2}) == [(0, None), (1, None)]


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_oracle_continues_from_any_cut(name):
    m, toks = oracle(name), [int(x) for x in tokens(name, 8, 23)[0]]
    whole = oracle_logits(name, tuple(toks))
    st, got, at = m.new_state(), [], 0
    for n in (1, 2, 7, 1, 1, 8, 3):
        got.append(m.fwd(toks[at:at + n], st))
        at += n
    assert at == 23 and np.max(np.abs(np.concatenate(got) - whole)) < 1e-9


class _Without(Z.Model):
    """The oracle with one mechanism left out: what the test models have to be able to tell apart."""

    def __init__(self, name, what):
        cfg = CONFIGS[name].to_dict()
        super().__init__(cfg, synth.llama_weights_f32(weights(name)))
        for l in cfg["layers"]:
            if what == "rotation":
                l["mixer"]["left"]["rot"] = {"dims": 0, "base": 1.0}
            if what == "scales":
                l["mixer"]["left_scale"] = l["mixer"]["right_scale"] = 1.0
            if what == "second expert" and l["mlp"] and l["mlp"]["kind"] == "moe":
                l["mlp"]["router"]["top"] = 1
            if what == "shared expert" and l["mlp"]:
                l["mlp"].pop("shared", None)
        if what == "soft cap":
            cfg["logit_softcap"] = None
        if what == "last pass":
            cfg["loop"]["times"] -= 1
            self.runs = Z.layer_runs(cfg)
        zero = {"oldest tap": ("mix.right.conv", lambda a: a[:, :1]), "convolution bias": ("mix.right.conv.b", lambda a: a),
                "step bias": ("mix.right.dt.b", lambda a: a), "step rank": ("mix.right.dt", lambda a: a),
                "skip": ("mix.right.D", lambda a: a), "token input": ("side.norm", lambda a: a), "step vector": ("step", lambda a: a),
                "router": ("mlp.router", lambda a: a)}
        for k in list(self.w):
            if what in zero and k.split(".", 1)[-1] == zero[what][0]:
                self.w[k] = self.w[k].copy()
                zero[what][1](self.w[k])[...] = 0.0
            if what == "embedding in the loop" and k == "loop.in":
                self.w[k] = self.w[k].copy()
                self.w[k][:, cfg["width"]:] = 0.0
            if what == "norm gain" and k.endswith(".norm1"):
                self.w[k] = np.ones_like(self.w[k])


@pytest.mark.parametrize("name", ["mixed", "odd"])
@pytest.mark.parametrize("what", ["rotation", "scales", "second expert", "shared expert", "soft cap", "last pass", "oldest tap",
                                  "convolution bias", "step bias", "step rank", "skip", "token input", "step vector", "router",
                                  "embedding in the loop", "norm gain"])
def test_models_show_a_missing_mechanism(name, what):
    """A mechanism left out moves the logits by more than the GPU tests allow in bf16, let alone in f32."""
    toks = tuple(int(x) for x in tokens(name, 9, 24)[0])
    m = _Without(name, what)
    assert logit_err(m.fwd(list(toks), m.new_state()), oracle_logits(name, toks)) > 0.1


class _Weighted(Z.Model):
    """Scores that weigh the experts' outputs instead of their inputs, or that are normalised to one."""
    how = "output"

    def _mlp(self, p, mlp, h):
        if mlp.get("kind") != "moe":
            return super()._mlp(p, mlp, h)
        w, out = self.w, np.zeros_like(h)
        three = lambda q: (w[q + "gate"], w[q + "up"], w[q + "down"])
        for i, z in enumerate(h @ w[p + "router"].T):
            chosen, s = Z.route(z, mlp["router"]["top"])
            if self.how == "normalised":
                s = s / s.sum()
            for e, f in zip(chosen, s):
                out[i] += Z.gated(f * h[i], *three(f"{p}e{e}.")) if self.how == "normalised" else f * Z.gated(h[i], *three(f"{p}e{e}."))
        return out + (Z.gated(h, *three(p + "shared.")) if mlp.get("shared") else 0.0)


@pytest.mark.parametrize("how", ["output", "normalised"])
def test_models_show_how_experts_are_weighted(how):
    toks = tuple(int(x) for x in tokens("mixed", 9, 24)[0])
    m = _Weighted(CONFIGS["mixed"].to_dict(), synth.llama_weights_f32(weights("mixed")))
    m.how = how
    assert logit_err(m.fwd(list(toks), m.new_state()), oracle_logits("mixed", toks)) > 0.1


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_models_show_a_lost_state(name):
    """A sequence whose state is dropped at a cut is told apart at once; so are passes that share one state."""
    toks = [int(x) for x in tokens(name, 10, 24)[0]]
    want = oracle_logits(name, tuple(toks))
    m = oracle(name)
    for key in ("k", "v", "conv", "s"):
        st = m.new_state()
        m.fwd(toks[:16], st)
        for run in st["runs"]:
            run[key] = run[key] * 0.0
        assert logit_err(m.fwd(toks[16:17], st), want[16:17]) > 0.1, key
    st = m.new_state()
    m.fwd(toks[:16], st)
    again = [n for n, (i, _) in enumerate(m.runs) if [j for j, _ in m.runs].index(i) < n]
    for n in again:
        first = [j for j, _ in m.runs].index(m.runs[n][0])
        st["runs"][n] = dict(st["runs"][first])
    assert again and logit_err(m.fwd(toks[16:17], st), want[16:17]) > 0.1


def test_config_round_trip_and_shapes():
    for cfg in CONFIGS.values():
        again = ZC.Config.from_dict(json.loads(json.dumps(cfg.to_dict())))
        assert again == cfg
        shapes = ZC.weight_shapes(cfg)
        assert list(shapes) == ZC.weight_names(cfg)
        assert ("loop.in" in shapes) == (cfg.loop is not None) and ("side.embed" in shapes) == (cfg.side_dim > 0)
        for i, l in enumerate(cfg.layers):
            assert (f"l{i}.mlp.router" in shapes) == isinstance(l.mlp, ZC.Experts)
            assert (f"l{i}.mlp.up" in shapes) == isinstance(l.mlp, int)
            assert shapes[f"l{i}.mix.right.x"][0] == l.right.dt_rank + 2 * l.right.state
    for change in (lambda l: l.update(type="other"), lambda l: l["mlp"].update(kind="other")):
        bad = CONFIGS["mixed"].to_dict()
        change(bad["layers"][0])
        with pytest.raises(ValueError):
            ZC.Config.from_dict(bad)


def test_registry_names_the_architecture():
    from ug_b200 import registry
    assert registry.architecture(CONFIGS["odd"].to_dict()) == "Zidevik"
    assert len(registry.DTYPES["Zidevik"]) == 2
