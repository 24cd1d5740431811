"""GPU parity of whole Zidevik models against oracle/zidevik_ref.py: prompts, token-by-token decoding, portions, batches,
sequences that follow one another, generation and trace replay through the package's own entry points.

Tolerances in zidevik_cases.LIMITS; test_zidevik_cpu.py shows that a missing mechanism or a lost state moves the test
models' logits by more than both, and everything runs in f32 too, where the limit is rounding at 2e-5."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from conftest import ROOT
from ug_b200 import DType, UgError, synth
from ug_b200.generate import generate
from ug_b200.zidevik import Config, Model
from zidevik_cases import CONFIGS, agree, layer, oracle, oracle_logits, position_err, reference, tokens, weights, write_model

pytestmark = pytest.mark.gpu
BOTH = [DType.F32, DType.BF16]


@pytest.fixture
def make(dev):
    made = []

    def f(name, dtype, batch=1, t_max=320, seed=500, **options):
        m = Model.new(CONFIGS[name], weights(name, seed), dev, batch, t_max, dtype)
        for k, v in options.items():
            m.set_option(k, v)
        made.append(m)
        return m
    yield f
    for m in made:
        m.close()


def want_of(name, row):
    return oracle_logits(name, tuple(int(x) for x in row))


def feed(m, row, cuts):
    """Logits of every position of one sequence fed in portions (1 = a decode step)."""
    out, at = [], 0
    for n in cuts:
        part = np.array([row[at:at + n]], np.int32)
        m.fwd(part)
        out.append(m.logits() if n == 1 else m.prefill_logits()[0])
        at += n
    assert at == len(row)
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt(make, name, dtype):
    m = make(name, dtype)
    for n in (1, 2, 40, 150):
        row = tokens(name, 40, n)[0]
        m.reset()
        m.prefill(row[None], all_logits=True)
        assert m.position == n
        want = want_of(name, row)
        assert agree(m.prefill_logits()[0], want, dtype == DType.F32)
        assert agree(m.logits(), want[-1:], dtype == DType.F32)
        assert m.next_tokens()[0] == int(np.argmax(m.logits()[0]))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_stream_after_every_layer_run(make, name):
    row = tokens(name, 41, 45)[0]
    m = make(name, DType.F32, keep_layers=1)
    m.prefill(row[None], all_logits=True)
    o, layers = oracle(name), []
    o.fwd([int(x) for x in row], o.new_state(), layers)
    want = np.stack(layers)
    assert m.layer_runs == len(layers)
    assert np.max(np.abs(m.layer_outputs()[:, 0] - want)) < 2e-5 * np.max(np.abs(want))


def test_unset_routing_in_32_bits(dev):
    """Routers that read the whole stream, with nothing done to keep the choices apart."""
    cfg = CONFIGS["wide_heads"]
    w = synth.zidevik_weights(cfg, 700)
    row = tokens("wide_heads", 57, 60)[0]
    ref = reference(cfg, w)
    m = Model.new(cfg, w, dev, 1, 64, DType.F32)
    m.prefill(row[None, :50], all_logits=True)
    got = [m.prefill_logits()[0]]
    for i in range(50, 60):
        m.fwd(row[i:i + 1])
        got.append(m.logits())
    m.close()
    assert agree(np.concatenate(got), ref.fwd(row, ref.new_state()), True)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_token_by_token(make, name, dtype):
    """From the first token on, and after a prompt; across the 16- and 64-position tiles of the attention kernels."""
    row = tokens(name, 42, 80)[0]
    want = want_of(name, row)
    m = make(name, dtype)
    assert agree(feed(m, row, [1] * 80), want, dtype == DType.F32)
    m.reset()
    assert agree(feed(m, row, [31] + [1] * 49), want, dtype == DType.F32)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name,cuts", [
    ("mixed", [2] * 10 + [3] * 5 + [1, 4, 1, 5, 64, 30]), ("mixed", [64, 63, 2, 1, 10]), ("odd", [2, 2, 17, 16, 1, 1, 101]),
    ("wide_heads", [65, 2, 2, 1, 50, 20]), ("plain", [5, 40, 1, 1, 2, 91]), ("once", [33, 2, 1, 70, 34]), ("mixed", [17, 16, 2, 1, 104])])
def test_portions(make, name, dtype, cuts):
    row = tokens(name, 43, sum(cuts))[0]
    assert agree(feed(make(name, dtype), row, cuts), want_of(name, row), dtype == DType.F32)


@pytest.mark.parametrize("dtype", BOTH)
def test_prompt_in_engine_chunks(make, dtype):
    """prefill_rows cuts one long call into chunks; which attention kernel takes short blocks must not matter."""
    row = tokens("mixed", 44, 150)[0]
    want = want_of("mixed", row)
    for rows, short in ((16, 16), (40, 0), (40, 64), (17, 3)):
        m = make("mixed", dtype, prefill_rows=rows, absorb_max=short)
        m.prefill(row[None], all_logits=True)
        assert agree(m.prefill_logits()[0], want, dtype == DType.F32)
        m.decode(1)
        row2 = np.append(row, np.int32(np.argmax(m.prefill_logits()[0, -1])))
        assert agree(m.logits(), want_of("mixed", row2)[-1:], dtype == DType.F32)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("batch", [3, 70])
def test_batch_rows_are_independent(make, dtype, batch):
    """Different sequences in one batch, in a prompt, a continued prompt and steps; the same as each alone."""
    rows = tokens("mixed", 45, 60, batch)
    m = make("mixed", dtype, batch, 96)
    m.prefill(rows[:, :37], all_logits=True)
    a = m.prefill_logits()
    m.prefill(rows[:, 37:57], all_logits=True)
    b = m.prefill_logits()
    steps = []
    for i in range(57, 60):
        m.fwd(rows[:, i])
        steps.append(m.logits())
    for k in {0, 1, batch - 1}:
        got = np.concatenate([a[k], b[k], np.stack([s[k] for s in steps])])
        assert agree(got, want_of("mixed", rows[k]), dtype == DType.F32)
    alone = make("mixed", dtype, 1, 96)
    alone.prefill(rows[1:2, :57])
    assert agree(b[1, -1:], alone.logits().astype(np.float64), dtype == DType.F32, 2.0)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_sequences_follow_one_another(make, name, dtype):
    """A reset gives cache and state back: a short sequence after a long one, the same one again, one that is only
    decoded, and a state that was left in the middle."""
    m = make(name, dtype)
    for seed, n, cuts in ((46, 200, [200]), (47, 3, [3]), (48, 35, [1] * 35), (46, 200, [150, 2, 48]), (49, 2, [2]), (48, 35, [20, 15])):
        row = tokens(name, seed, n)[0]
        m.reset()
        assert agree(feed(m, row, cuts), want_of(name, row), dtype == DType.F32)
    m.prefill(tokens(name, 50, 21))               # abandoned here
    row = tokens(name, 47, 3)[0]
    m.reset()
    assert agree(feed(m, row, [1, 1, 1]), want_of(name, row), dtype == DType.F32)
    with pytest.raises(UgError):
        m.reset(1)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("n", [33, 64, 65, 129, 257])
def test_far_keys(dev, dtype, n):
    """Attention alone with sharp scores: token 5 occurs once, at the start or at a tile border, and draws the attention of every
    later position, in a prompt and decoded."""
    cfg = Config(vocab=64, width=64, eps=1e-5, layers=[layer((2, 1, 32, 16, 8, 1e6, 1.5), (8, 8, 1, 8), None)])
    w = {k: synth.bf16_bits_to_f32(v).copy() for k, v in synth.zidevik_weights(cfg, 77).items()}
    w["l0.mix.right.o"][:] = 0.0
    bits = {k: synth.to_bf16_bits(v) for k, v in w.items()}
    ref = reference(cfg, bits)
    m = Model.new(cfg, bits, dev, 1, 288, dtype)
    for at in sorted({0, 1, 15, 16, 31, n // 2, n - 2}):
        row = 8 + synth.tokens(at, (n,), 6)
        row[at] = 5
        want = ref.fwd([int(x) for x in row], ref.new_state())
        plain = row.copy()
        plain[at] = 8
        if at < n - 2:                            # the one token shows in what later positions compute
            assert np.max(position_err(ref.fwd([int(x) for x in plain], ref.new_state())[at + 1:], want[at + 1:])) > 0.03
        for cuts in ([n], [n - 20] + [1] * 20):
            m.reset()
            assert agree(feed(m, row, cuts), want, dtype == DType.F32, 3.0)
    m.close()


@pytest.mark.parametrize("dtype", BOTH)
def test_scan_reaches_back_to_the_first_token(dev, dtype):
    """The scan alone, with channels that hardly forget: the first token still shows hundreds of positions later, however the
    prompt is cut; a state that starts anew at a cut would show too."""
    cfg = Config(vocab=64, width=64, eps=1e-5, layers=[layer((1, 1, 8, 8, 8, 100.0, 0.3), (64, 16, 4, 8), None)])
    w = {k: synth.bf16_bits_to_f32(v).copy() for k, v in synth.zidevik_weights(cfg, 78).items()}
    w["l0.mix.left.o"][:] = 0.0
    w["l0.mix.right.A_log"][:] = -8.0
    bits = {k: synth.to_bf16_bits(v) for k, v in w.items()}
    ref, n = reference(cfg, bits), 260
    row = synth.tokens(3, (n,), 64)
    other = row.copy()
    other[0] = (row[0] + 7) % 64
    want = ref.fwd(row, ref.new_state())
    assert np.max(position_err(ref.fwd(other, ref.new_state())[-20:], want[-20:])) > 0.01
    st = ref.new_state()
    ref.fwd(row[:130], st)
    st["runs"][0]["s"] *= 0.0
    assert np.max(position_err(ref.fwd(row[130:], st), want[130:])) > 0.1
    m = Model.new(cfg, bits, dev, 1, 288, dtype)
    for cuts in ([n], [130, 130], [2] * 20 + [220], [n - 40] + [1] * 40):
        m.reset()
        assert agree(feed(m, row, cuts), want, dtype == DType.F32)
    m.close()


@pytest.mark.parametrize("dtype", BOTH)
def test_long_decoding(make, dtype):
    """400 steps, logits checked now and then against the oracle that is fed the same tokens."""
    m = make("odd", dtype, t_max=512)
    o = oracle("odd")
    row = [int(x) for x in tokens("odd", 51, 12)[0]]
    m.prefill(np.array([row], np.int32))
    st = o.new_state()
    o.fwd(row, st)
    for i in range(400):
        tok = int(m.next_tokens()[0])
        m.decode(1)
        want = o.fwd([tok], st)
        if i % 57 == 0 or i == 399:
            assert agree(m.logits(), want, dtype == DType.F32)
    assert m.position == 412


@pytest.mark.parametrize("pdl", [0, 1])
@pytest.mark.parametrize("splits", [0, 1, 5, 8])
def test_options_do_not_change_results(make, pdl, splits):
    row = tokens("wide_heads", 52, 90)[0]
    m = make("wide_heads", DType.BF16, pdl=pdl, att_splits=splits)
    assert agree(feed(m, row, [70] + [1] * 20), want_of("wide_heads", row), False)


def test_greedy_generation(make):
    """generate() against the oracle's argmax in f32, whole and in portions, and the same tokens for a row in a batch."""
    rows = tokens("mixed", 53, 20, 4)
    want = []
    o = oracle("mixed")
    for r in rows:
        st = o.new_state()
        logits, seq = o.fwd([int(x) for x in r], st)[-1], []
        for _ in range(12):
            seq.append(int(np.argmax(logits)))
            logits = o.fwd([seq[-1]], st)[-1]
        want.append(seq)
    m = make("mixed", DType.F32, 4, 64)
    assert generate(m, rows, 12).tolist() == want
    assert generate(m, rows, 12, chunk=7).tolist() == want
    one = make("mixed", DType.F32, 1, 64)
    assert generate(one, rows[2:3], 12, chunk=2).tolist() == want[2:3]
    with pytest.raises(UgError):
        generate(one, rows[:1], 60)                # more than the cache holds
    with pytest.raises(UgError):
        generate(one, rows, 4)


def test_bad_token_is_reported(make, dev):
    m = make("odd", DType.BF16)
    m.prefill(np.array([[1, 2, CONFIGS["odd"].vocab, 3]], np.int32))
    with pytest.raises(UgError):
        dev.synchronize()
    m.reset()
    row = tokens("odd", 54, 9)[0]
    assert agree(feed(m, row, [9]), want_of("odd", row), False)


def test_wrong_shapes_and_names_are_rejected(dev):
    cfg = CONFIGS["odd"]
    w = dict(weights("odd"))
    w["l1.mlp.e2.up"] = w["l1.mlp.e2.up"][:-1]
    with pytest.raises(ValueError):
        Model.new(cfg, w, dev, 1, 32)
    m = Model(cfg, dev, 1, 32)
    for name in ("l9.norm1", "l1.norm2", "l0.mlp.router", "l1.mlp.gate", "l1.mlp.e3.up", "l1.mlp.e1x.up", "lx.norm1", "embed.norm", "norm"):
        with pytest.raises(UgError):
            m.load_weight(name, weights("odd")["final.norm"])
    m.close()
    with pytest.raises(UgError):
        Model(cfg, dev, 500, 32)


def test_folder_registry_command_and_trace(dev, tmp_path):
    """A model folder through the registry, the generation command and the trace runner (own processes)."""
    from ug_b200 import registry
    folder = tmp_path / "model"
    folder.mkdir()
    write_model(folder, CONFIGS["mixed"], weights("mixed"))
    row = [int(x) for x in tokens("mixed", 55, 30)[0]]
    m = registry.load(str(folder), dev, 1, 64, DType.F32)
    assert isinstance(m, Model) and m.state_bytes(10) > 0
    ids = generate(m, np.array([row], np.int32), 8)[0].tolist()
    m.close()
    r = subprocess.run([sys.executable, "-m", "ug_b200.generate", "--model", str(folder), "--prompt", ",".join(map(str, row)),
                        "-n", "8", "--chunk", "11", "--dtype", "float32"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split() == [",".join(map(str, ids))]
    other = [int(x) for x in tokens("mixed", 56, 9)[0]]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": row[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": row[20:21], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": row[21:], "want": []}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": other, "want": [8]}], "end": ["b"]}]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), cwd=str(tmp_path),
                           capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
        assert sorted(os.listdir(out)) == ["0.f32", "1.f32", "3.f32"]
        want, second = want_of("mixed", row), want_of("mixed", other)
        for step, rows in ((0, want[[0, 19]]), (1, want[[20]]), (3, second[[8]])):
            got = np.fromfile(out / f"{step}.f32", "<f4").reshape(-1, CONFIGS["mixed"].vocab)
            assert agree(got, rows, dtype == "float32")
