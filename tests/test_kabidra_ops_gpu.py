"""GPU parity of each Kabidra mechanism alone, through the C ABI, against the plain equations of oracle/kabidra_ref.py."""
import numpy as np
import pytest

from hybrid_cases import Buf, close
from oracle import kabidra_ref as K
from ug_b200 import UgError, synth

pytestmark = pytest.mark.gpu


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("taps,width,batch,cuts", [
    (1, 8, 2, (5,)), (2, 24, 1, (1, 1, 2, 9)), (3, 1032, 2, (8, 7, 1, 30)), (4, 200, 3, (2, 1, 16, 17)), (7, 16, 2, (1, 2, 3, 4, 40))])
def test_causal_conv(dev, bf16, taps, width, batch, cuts):
    """Blocks of any size, shorter than the taps too, continue one another."""
    B, t = Buf(dev, bf16), sum(cuts)
    h = synth.normal(1, (batch, t, width))
    w = synth.normal(2, (width, taps), 0.5)
    _, hv = B.act(h)
    tail, _ = B.act(np.zeros((batch, max(taps - 1, 1), width)))
    ws = B.f32(w.T)
    want = np.stack([hv[b] + K.causal_conv(hv[b], w.astype(np.float64), np.zeros((taps - 1, width)))[0] for b in range(batch)])
    at = 0
    for n in cuts:
        hs, _ = B.act(h[:, at:at + n])
        out = B.out(batch * n * width)
        dev.causal_conv(hs, ws, tail, out, batch, n, width, taps)
        assert close(B.read(out, (batch, n, width)), want[:, at:at + n], B.tol)
        at += n
    if taps > 1:
        assert np.array_equal(B.read(tail, (batch, taps - 1, width)), hv[:, t - taps + 1:])


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("width,batch,cuts", [
    (8, 1, (1, 2, 7, 8, 9)), (40, 3, (127, 1, 128, 129)), (320, 2, (1000, 1, 1)), (2048, 1, (300, 2)), (64, 1, (2500, 1, 1100)), (32, 20, (260,))])
def test_min_gru(dev, bf16, width, batch, cuts):
    """The scan over blocks and single steps, the state carried between them; slow decay so that far inputs stay
    visible, pre-activations on both sides of the candidate's branch."""
    B, t = Buf(dev, bf16), sum(cuts)
    pre = synth.normal(3, (batch, t, 3, width), 1.5)
    pre[:, :, 0] -= 3.0
    bz, bx = synth.normal(4, (width,)), synth.normal(5, (width,))
    state0 = synth.normal(6, (batch, width))
    z = K.sigmoid(pre[:, :, 0].astype(np.float64) + bz)
    c = K.gru_candidate(pre[:, :, 1].astype(np.float64) + bx)
    S = np.stack([K.min_gru(z[b], c[b], state0[b].astype(np.float64))[0] for b in range(batch)])
    want = S * K.silu(pre[:, :, 2].astype(np.float64))
    st, zs, xs, at = B.f32(state0), B.f32(bz), B.f32(bx), 0
    for n in cuts:
        out = B.out(batch * n * width)
        dev.min_gru(B.f32(pre[:, at:at + n]), zs, xs, st, out, batch, n, width)
        assert close(B.read(out, (batch, n, width)), want[:, at:at + n], B.tol)
        at += n
        assert close(st.to_vec().reshape(batch, width).astype(np.float64), S[:, at - 1], 2e-5)


@pytest.mark.parametrize("width,batch,cuts", [(8, 2, (2, 3, 64, 65)), (72, 1, (511, 512, 513)), (2048, 2, (700,))])
def test_min_gru_on_bf16_projections(dev, width, batch, cuts):
    """A block whose pre-activations were rounded to bf16: the recurrence itself stays in 32 bits."""
    B, t = Buf(dev, True), sum(cuts)
    pre = synth.normal(3, (batch, t, 3, width), 1.5)
    pre[:, :, 0] -= 3.0
    bz, bx = synth.normal(4, (width,)), synth.normal(5, (width,))
    st, zs, xs, at = B.f32(np.zeros((batch, width))), B.f32(bz), B.f32(bx), 0
    S0 = np.zeros((batch, width))
    for n in cuts:
        ps, pv = B.act(pre[:, at:at + n])
        out = B.out(batch * n * width)
        dev.min_gru(ps, zs, xs, st, out, batch, n, width)
        z, c = K.sigmoid(pv[:, :, 0] + bz), K.gru_candidate(pv[:, :, 1] + bx)
        S = np.stack([K.min_gru(z[b], c[b], S0[b])[0] for b in range(batch)])
        S0 = S[:, -1]
        assert close(B.read(out, (batch, n, width)), S * K.silu(pv[:, :, 2]), B.tol)
        assert close(st.to_vec().reshape(batch, width).astype(np.float64), S0, 2e-5)
        at += n


def test_min_gru_remembers_the_first_token(dev):
    """With the gate shut after position 0 the state is the first candidate for as long as anyone looks."""
    B, n, width = Buf(dev, False), 3000, 40
    pre = np.zeros((1, n, 3, width), np.float32)
    pre[:, 0, 0] = 30.0
    pre[:, 0, 1] = synth.normal(7, (width,))
    pre[:, 1:, 0] = -40.0
    pre[:, :, 2] = 1.0
    st, zero, out = B.f32(np.zeros(width)), B.f32(np.zeros(width)), B.out(n * width)
    dev.min_gru(B.f32(pre), zero, zero, st, out, 1, n, width)
    first = K.gru_candidate(pre[0, 0, 1].astype(np.float64))
    assert np.allclose(st.to_vec(), first, rtol=1e-5, atol=1e-6)
    assert np.allclose(B.read(out, (n, width)), first * K.silu(1.0), rtol=1e-5, atol=1e-6)


def latent_want(q, c, gate, scale, pos0):
    t, heads, rank = q.shape
    out = np.empty_like(q)
    for i in range(t):
        for h in range(heads):
            p = K.softmax(c[:pos0 + i + 1] @ q[i, h] * scale)
            out[i, h] = (p @ c[:pos0 + i + 1]) * (1.0 if gate is None else gate[i, h])
    return out


@pytest.mark.parametrize("bf16,rank", [(False, 8), (False, 72), (False, 560), (True, 64), (True, 128), (True, 256), (True, 384), (True, 512), (True, 72), (True, 560)])
@pytest.mark.parametrize("heads,batch,t,pos0,slices", [(3, 2, 1, 31, 1), (16, 1, 1, 32, 3), (17, 2, 3, 62, 2), (1, 1, 2, 0, 1), (40, 1, 1, 300, 7)])
def test_latent_attention(dev, bf16, rank, heads, batch, t, pos0, slices):
    B, t_max = Buf(dev, bf16), 320
    q, qv = B.act(synth.normal(8, (batch, t, heads, rank)))
    c, cv = B.act(synth.normal(9, (batch, t_max, rank)))
    gate = K.sigmoid(synth.normal(10, (batch, t, heads))).astype(np.float32)
    scale = 2.0 / rank ** 0.5
    out, pos = B.out(batch * t * heads * rank), dev.slice_from_values(np.array([pos0], np.int32))
    dev.latent_attend(q, c, B.f32(gate), pos, out, batch, t, heads, rank, t_max, scale, slices)
    dev.synchronize()
    got = B.read(out, (batch, t, heads, rank))
    for b in range(batch):
        assert close(got[b], latent_want(qv[b], cv[b], gate[b].astype(np.float64), scale, pos0), 2e-2 if bf16 else 2e-5)


@pytest.mark.parametrize("bf16,rank", [(False, 64), (True, 64), (True, 128), (True, 512), (True, 384)])
@pytest.mark.parametrize("last,far", [(0, 0), (31, 0), (32, 0), (32, 31), (32, 32), (63, 32), (64, 63), (257, 0), (257, 255), (257, 256), (511, 257)])
def test_latent_attention_finds_one_key(dev, bf16, rank, last, far):
    """One key stands out by a score of 40: the output is that key's latent, at every tile and slice border; the same
    key one position after the query changes nothing."""
    B, t_max, heads = Buf(dev, bf16), 512, 2
    c = 0.05 * synth.normal(11, (1, t_max, rank))
    c[0, far, :] = 0.0
    c[0, far, 5] = 4.0
    if last + 1 < t_max:
        c[0, last + 1, :] = 0.0
        c[0, last + 1, 5] = 100.0                      # not visible
    q = np.zeros((1, 1, heads, rank), np.float32)
    q[..., 5] = 10.0
    cs, cv = B.act(c)
    qs, qv = B.act(q)
    for slices in (1, 2, 5):
        out, pos = B.out(heads * rank), dev.slice_from_values(np.array([last], np.int32))
        dev.latent_attend(qs, cs, None, pos, out, 1, 1, heads, rank, t_max, 1.0, slices)
        got = B.read(out, (heads, rank))
        want = np.zeros(rank)
        want[5] = 4.0
        assert np.max(np.abs(got - want)) < 0.02
        assert close(got, latent_want(qv[0], cv[0], None, 1.0, last)[0], 1e-2)


def test_latent_attention_rejects_a_position_outside_the_cache(dev):
    B = Buf(dev, True)
    q, c, out = B.out(64), B.act(np.zeros((1, 32, 64)))[0], B.out(64)
    q.copy_host_to_device(np.zeros(64, np.uint16), bf16=True)
    pos = dev.slice_from_values(np.array([32], np.int32))
    dev.latent_attend(q, c, None, pos, out, 1, 1, 1, 64, 32, 1.0)
    with pytest.raises(UgError):
        dev.synchronize()
    dev.synchronize()


@pytest.mark.parametrize("dq,dv", [(64, 64), (64, 128), (128, 64), (128, 128)])
@pytest.mark.parametrize("batch,t,pos0,heads", [(1, 1, 0, 1), (2, 130, 0, 3), (1, 64, 63, 2), (1, 300, 65, 5), (2, 17, 200, 2)])
def test_causal_attention_wide(dev, dq, dv, batch, t, pos0, heads):
    B, n = Buf(dev, True), pos0 + t
    q, qv = B.act(synth.normal(12, (batch, t, heads, dq)))
    k, kv = B.act(synth.normal(13, (batch, n, heads, dq)))
    v, vv = B.act(synth.normal(14, (batch, n, heads, dv)))
    gate = K.sigmoid(synth.normal(15, (batch, t, heads))).astype(np.float32)
    out, scale = B.out(batch * t * heads * dv), 2.0 / dq ** 0.5
    dev.causal_attention_wide(q, k, v, B.f32(gate), out, batch, t, pos0, heads, dq, dv, scale)
    dev.synchronize()
    got = B.read(out, (batch, t, heads, dv))
    mask = np.arange(n)[None, :] > pos0 + np.arange(t)[:, None]
    for b in range(batch):
        for h in range(heads):
            s = qv[b, :, h] @ kv[b, :, h].T * scale
            want = K.softmax(np.where(mask, -np.inf, s)) @ vv[b, :, h] * gate[b, :, h:h + 1]
            assert close(got[b, :, h], want, 2e-2)


@pytest.mark.parametrize("dq,dv", [(64, 128), (128, 128)])
def test_causal_attention_wide_finds_one_key(dev, dq, dv):
    """Query i looks for a key only key i has (and for none of its own future): the diagonal, one position off it and
    keys at tile borders."""
    B, t = Buf(dev, True), 260
    k = 0.01 * synth.normal(16, (1, t, 1, dq))
    v = synth.normal(17, (1, t, 1, dv))
    q = np.zeros((1, t, 1, dq), np.float32)
    target = [i if i % 3 == 0 else (max(0, i - 1) if i % 3 == 1 else (i // 64) * 64) for i in range(t)]
    codes = synth.normal(18, (t, dq))
    codes /= np.linalg.norm(codes, axis=1, keepdims=True)
    k[0, :, 0] += codes
    for i in range(t):
        q[0, i, 0] = 60.0 * codes[target[i]]
    (qs, qv), (ks, kv), (vs, vv) = B.act(q), B.act(k), B.act(v)
    out = B.out(t * dv)
    dev.causal_attention_wide(qs, ks, vs, None, out, 1, t, 0, 1, dq, dv, 1.0)
    got = B.read(out, (t, dv))
    mask = np.arange(t)[None, :] > np.arange(t)[:, None]
    want = K.softmax(np.where(mask, -np.inf, qv[0, :, 0] @ kv[0, :, 0].T)) @ vv[0, :, 0]
    assert np.max(np.abs(got - want)) < 0.05


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("rows,width,n", [(3, 8, 0), (5, 200, 1), (2, 1024, 7), (4, 2048, 23), (1, 4096, 9), (1, 8192, 5), (2, 1032, None)])
def test_residual_update(dev, bf16, rows, width, n):
    B = Buf(dev, bf16)
    x, y = synth.normal(19, (rows, width)), synth.normal(20, (rows, width), 3.0)
    pg, g = synth.uniform(21, (width,), -0.5, 1.5), synth.uniform(22, (width,), -0.5, 1.5)
    f = np.float64
    res = x.astype(f) + K.rms(y.astype(f), 1e-3) * pg.astype(f)
    bank = dwa = None
    want = res
    if n is not None:
        hist = synth.normal(23, (n, rows, width))
        co = synth.normal(24, (n + 1,))
        want = K.depth_average(co.astype(f), list(hist.astype(f)) + [res])
        bank, dwa = B.f32(np.concatenate([hist, np.zeros((1, rows, width), np.float32)])), B.f32(co)
    xs, h = B.f32(x), B.out(rows * width)
    dev.residual_update(xs, B.f32(y), B.f32(pg), bank, dwa, n or 0, B.f32(g), h, rows, width, 1e-3)
    assert close(xs.to_vec().reshape(rows, width).astype(f), want, 2e-6)
    assert close(B.read(h, (rows, width)), K.rms(want, 1e-3) * g.astype(f), B.tol)
    if bank is not None:
        assert close(bank.to_vec().reshape(n + 1, rows, width)[n].astype(f), res, 2e-6)
