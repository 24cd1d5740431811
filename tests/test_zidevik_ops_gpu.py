"""GPU parity of each Zidevik mechanism alone: through the C ABI against the plain equations of oracle/zidevik_ref.py, and for
what has no operator of its own through models that consist of that mechanism."""
import numpy as np
import pytest

from hybrid_cases import Buf, close
from oracle import zidevik_ref as Z
from ug_b200 import DType, UgError, synth
from ug_b200.zidevik import Config, Experts, Loop, Model
from zidevik_cases import layer, reference, separate_experts

pytestmark = pytest.mark.gpu
f64 = np.float64


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("taps,width,batch,cuts", [
    (1, 8, 2, (5,)), (2, 24, 1, (1, 1, 2, 9)), (3, 1032, 2, (8, 7, 1, 30)), (4, 200, 3, (2, 1, 16, 17)), (7, 16, 2, (1, 2, 3, 4, 40))])
def test_gated_conv(dev, bf16, taps, width, batch, cuts):
    """Blocks of any size, shorter than the taps too, continue one another."""
    B, t = Buf(dev, bf16), sum(cuts)
    h, w, bias = synth.normal(1, (batch, t, width)), synth.normal(2, (width, taps), 0.5), synth.normal(3, (width,))
    _, hv = B.act(h)
    tail, _ = B.act(np.zeros((batch, max(taps - 1, 1), width)))
    ws, bs = B.f32(w.T), B.f32(bias)
    want = np.stack([Z.causal_conv(hv[b], w.astype(f64), bias.astype(f64), np.zeros((taps - 1, width)))[0] for b in range(batch)])
    at = 0
    for n in cuts:
        hs, _ = B.act(h[:, at:at + n])
        out = B.out(batch * n * width)
        dev.gated_conv(hs, ws, bs, tail, out, batch, n, width, taps)
        assert close(B.read(out, (batch, n, width)), want[:, at:at + n], B.tol)
        at += n
    if taps > 1:
        assert np.array_equal(B.read(tail, (batch, taps - 1, width)), hv[:, t - taps + 1:])


def half_split(x, pos, base, dims):
    """The other layout of the pairs, (i, i + dims / 2), by reordering the dimensions."""
    order = np.r_[np.arange(dims).reshape(2, dims // 2).T.ravel(), np.arange(dims, x.shape[2])]
    out = np.empty_like(x)
    out[:, :, order] = Z.rotate(x[:, :, order], pos, base, dims)
    return out


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("interleaved,norm", [(1, 1), (0, 1), (1, 0)])
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,batch,t,pos0", [
    (2, 1, 8, 8, 8, 1, 3, 0), (6, 3, 64, 128, 16, 2, 5, 31), (4, 4, 72, 24, 72, 1, 2, 990), (3, 1, 256, 40, 128, 2, 1, 63), (5, 5, 40, 16, 0, 1, 4, 7)])
def test_rotated_heads_and_cache_append(dev, bf16, interleaved, norm, heads, kv, dim, vdim, rot, batch, t, pos0):
    B, t_max, eps, base = Buf(dev, bf16), 1024, 1e-3, 500.0
    ld = (heads + kv) * dim + kv * vdim
    pre, pv = B.act(synth.normal(4, (batch, t, ld), 2.0))
    angle = np.arange(t_max)[:, None] * base ** (-2.0 * np.arange(max(rot // 2, 1)) / max(rot, 1))
    q = B.out(batch * t * heads * dim)
    kc, k0 = B.act(synth.normal(5, (batch, kv, t_max, dim)))
    vc, v0 = B.act(synth.normal(6, (batch, kv, t_max, vdim)))
    dev.head_inputs(pre, B.f32(np.cos(angle)), B.f32(np.sin(angle)), dev.slice_from_values(np.array([pos0], np.int32)), q, kc, vc, batch, t,
                    heads, kv, dim, vdim, rot, interleaved, norm, eps, t_max)
    turn = Z.rotate if interleaved else half_split
    for b in range(batch):
        x = pv[b, :, :(heads + kv) * dim].reshape(t, heads + kv, dim)
        x = turn(x, pos0 + np.arange(t), base, rot) if rot else x
        x = Z.rms(x, eps) if norm else x
        k0[b, :, pos0:pos0 + t] = x[:, heads:].transpose(1, 0, 2)
        v0[b, :, pos0:pos0 + t] = pv[b, :, (heads + kv) * dim:].reshape(t, kv, vdim).transpose(1, 0, 2)
        assert close(B.read(q, (batch, t, heads, dim))[b], x[:, :heads], B.tol)
    assert close(B.read(kc, k0.shape), k0, B.tol) and np.array_equal(B.read(vc, v0.shape), v0)


@pytest.mark.parametrize("bf16,dq,dv", [(False, 8, 16), (False, 72, 40), (False, 136, 200), (True, 64, 64), (True, 64, 128), (True, 128, 64),
                                        (True, 128, 128), (True, 72, 64), (True, 256, 136)])
@pytest.mark.parametrize("heads,kv,batch,t,pos0,slices", [(3, 3, 2, 1, 31, 1), (16, 1, 1, 1, 16, 3), (34, 2, 2, 3, 62, 2), (2, 1, 1, 2, 0, 1), (24, 8, 1, 1, 300, 7), (8, 4, 3, 1, 47, 8)])
def test_grouped_attention(dev, bf16, dq, dv, heads, kv, batch, t, pos0, slices):
    B, t_max, scale = Buf(dev, bf16), 320, 2.0 / dq ** 0.5
    q, qv = B.act(synth.normal(7, (batch, t, heads, dq)))
    k, kv_ = B.act(synth.normal(8, (batch, kv, t_max, dq)))
    v, vv = B.act(synth.normal(9, (batch, kv, t_max, dv)))
    out = B.out(batch * t * heads * dv)
    dev.grouped_attend(q, k, v, dev.slice_from_values(np.array([pos0], np.int32)), out, batch, t, heads, kv, dq, dv, t_max, scale, 0.7, slices)
    dev.synchronize()
    got = B.read(out, (batch, t, heads, dv))
    for b in range(batch):
        want = 0.7 * Z.grouped_attention(qv[b], kv_[b].transpose(1, 0, 2), vv[b].transpose(1, 0, 2), scale, pos0)
        assert close(got[b], want, 2e-2 if bf16 else 2e-5)


@pytest.mark.parametrize("bf16,d", [(False, 64), (True, 64), (True, 128)])
@pytest.mark.parametrize("last,far", [(0, 0), (15, 0), (16, 0), (16, 15), (16, 16), (63, 16), (64, 63), (257, 0), (257, 255), (257, 256), (511, 257)])
def test_grouped_attention_finds_one_key(dev, bf16, d, last, far):
    """One key stands out by a score of 40: the output is that key's value, at every piece and slice border; a stronger key one
    position after the query changes nothing."""
    B, t_max, heads = Buf(dev, bf16), 512, 4
    k, v = 0.05 * synth.normal(10, (1, 2, t_max, d)), synth.normal(11, (1, 2, t_max, d))
    k[:, :, :, 5] = 0.0
    k[:, :, far, 5] = 4.0
    if last + 1 < t_max:
        k[:, :, last + 1, 5] = 100.0                        # not visible
    q = np.zeros((1, 1, heads, d), np.float32)
    q[..., 5] = 10.0
    (qs, _), (ks, _), (vs, vv) = B.act(q), B.act(k), B.act(v)
    for slices in (1, 2, 5, 8):
        out = B.out(heads * d)
        dev.grouped_attend(qs, ks, vs, dev.slice_from_values(np.array([last], np.int32)), out, 1, 1, heads, 2, d, d, t_max, 1.0, 1.0, slices)
        got = B.read(out, (heads, d))
        assert np.max(np.abs(got - vv[0, :, far].repeat(2, axis=0))) < 0.03


def test_grouped_attention_rejects_a_position_outside_the_cache(dev):
    B = Buf(dev, True)
    q, k, v, out = B.act(np.zeros(64))[0], B.act(np.zeros((32, 64)))[0], B.act(np.zeros((32, 64)))[0], B.out(64)
    for n in (32, -1):
        dev.grouped_attend(q, k, v, dev.slice_from_values(np.array([n], np.int32)), out, 1, 1, 1, 1, 64, 64, 32, 1.0)
        with pytest.raises(UgError):
            dev.synchronize()
        dev.synchronize()


@pytest.mark.parametrize("dq,dv", [(64, 64), (64, 128), (128, 64), (128, 128)])
@pytest.mark.parametrize("batch,t,pos0,heads,kv", [(1, 1, 0, 2, 1), (2, 130, 0, 6, 2), (1, 64, 63, 4, 4), (1, 300, 65, 5, 1), (2, 17, 200, 4, 2)])
def test_grouped_attention_block(dev, dq, dv, batch, t, pos0, heads, kv):
    B, n, t_max, scale = Buf(dev, True), pos0 + t, 384, 2.0 / dq ** 0.5
    q, qv = B.act(synth.normal(12, (batch, t, heads, dq)))
    k, kk = B.act(synth.normal(13, (batch, kv, t_max, dq)))
    v, vv = B.act(synth.normal(14, (batch, kv, t_max, dv)))
    out = B.out(batch * t * heads * dv)
    dev.grouped_attend_block(q, k, v, out, batch, t, pos0, heads, kv, dq, dv, t_max, scale, 1.3)
    dev.synchronize()
    got = B.read(out, (batch, t, heads, dv))
    mask = np.arange(n)[None, :] > pos0 + np.arange(t)[:, None]
    for b in range(batch):
        for h in range(heads):
            s = qv[b, :, h] @ kk[b, h // (heads // kv), :n].T * scale
            want = 1.3 * Z.softmax(np.where(mask, -np.inf, s)) @ vv[b, h // (heads // kv), :n]
            assert close(got[b, :, h], want, 2e-2)


def scan_inputs(t, batch, channels, states):
    x, z = synth.normal(15, (batch, t, channels)), synth.normal(16, (batch, t, channels))
    dt, bc = synth.normal(17, (batch, t, channels)), synth.normal(18, (batch, t, 2 * states))
    a_log = synth.uniform(19, (channels, states), -5.0, 1.0)
    return x, dt, bc, z, a_log, synth.normal(20, (channels,)), synth.normal(21, (channels,)) - np.float32(2.0)


def scan_want(xv, dtv, bcv, zv, a_log, skip, bias, s0, scale):
    n = a_log.shape[1]
    y, s = Z.selective_scan(xv, Z.softplus(dtv + bias.astype(f64)), -np.exp(a_log.astype(f64)), bcv[:, :n], bcv[:, n:], skip.astype(f64), s0)
    return y * Z.silu(zv) * scale, s


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("channels,states,batch,cuts", [
    (8, 8, 2, (2, 3, 7)), (40, 16, 1, (31, 32, 33, 2)), (200, 24, 2, (64, 5)), (72, 32, 1, (9, 40)), (16, 48, 1, (70,)), (32, 64, 2, (33, 2)),
    (24, 128, 1, (2, 17, 8)), (8, 256, 1, (40,)), (264, 16, 1, (700, 2)), (512, 16, 10, (37, 3)), (264, 8, 20, (19, 2))])
def test_selective_scan(dev, bf16, channels, states, batch, cuts):
    """Blocks that continue one another from a given state, for every dealing of states to lanes, with few CTAs and with many."""
    B, t = Buf(dev, bf16), sum(cuts)
    x, dt, bc, z, a_log, skip, bias = scan_inputs(t, batch, channels, states)
    s0 = synth.normal(22, (batch, channels, states))
    state, S, at = B.f32(s0), s0.astype(f64), 0
    for n in cuts:
        (xs, xv), (ds, dv), (bs, bv), (zs, zv) = (B.act(q[:, at:at + n]) for q in (x, dt, bc, z))
        out = B.out(batch * n * channels)
        dev.selective_scan(xs, ds, bs, zs, B.f32(a_log), B.f32(skip), B.f32(bias), state, out, batch, n, channels, states, 0.8)
        got = B.read(out, (batch, n, channels))
        for b in range(batch):
            want, S[b] = scan_want(xv[b], dv[b], bv[b], zv[b], a_log, skip, bias, S[b], 0.8)
            assert close(got[b], want, B.tol)
        assert close(state.to_vec().reshape(S.shape).astype(f64), S, 5e-5 if bf16 else 1e-5)
        at += n


@pytest.mark.parametrize("bf16", [False, True])
@pytest.mark.parametrize("channels,states,rank,rows,steps", [
    (8, 8, 8, 1, 5), (40, 16, 24, 3, 4), (200, 24, 8, 4, 3), (72, 32, 136, 5, 3), (16, 48, 16, 2, 3), (32, 64, 200, 9, 2), (24, 128, 40, 6, 3), (8, 256, 8, 1, 3), (40, 16, 520, 3, 2), (72, 16, 136, 40, 2)])
def test_selective_step(dev, bf16, channels, states, rank, rows, steps):
    B = Buf(dev, bf16)
    w, wv = B.act(synth.normal(23, (rank, channels), rank ** -0.5))
    S = synth.normal(24, (rows, channels, states)).astype(f64)
    state = B.f32(S)
    for i in range(steps):
        x, _, _, z, a_log, skip, bias = scan_inputs(1, rows, channels, states)
        low = synth.normal(25 + i, (rows, rank + 2 * states))
        if bf16:                                            # the projection's operand is rounded, B and C are not
            low[:, :rank] = synth.bf16_bits_to_f32(synth.to_bf16_bits(low[:, :rank]))
        xs, xv = B.act(x[:, 0])
        out = B.out(rows * channels)
        dev.selective_step(xs, B.f32(low), w, B.f32(z[:, 0]), B.f32(a_log), B.f32(skip), B.f32(bias), state, out, rows, channels, rank, states, 1.2)
        got = B.read(out, (rows, channels))
        for r in range(rows):
            want, S[r] = scan_want(xv[r:r + 1], low[r:r + 1, :rank].astype(f64) @ wv, low[r:r + 1, rank:].astype(f64), z[r].astype(f64),
                                   a_log, skip, bias, S[r], 1.2)
            assert close(got[r], want[0], B.tol)
        assert close(state.to_vec().reshape(S.shape).astype(f64), S, 2e-5)


@pytest.mark.parametrize("bf16", [False, True])
def test_scan_remembers_the_first_token(dev, bf16):
    """A state that never decays: what the first position wrote is read for as long as anyone looks, and nothing else is."""
    B, n, ch, st = Buf(dev, bf16), 3000, 40, 16
    x, bc = np.zeros((1, n, ch), np.float32), np.zeros((1, n, 2 * st), np.float32)
    x[0, 0] = synth.normal(30, (ch,))
    bc[0, 0, :st] = 1.0
    bc[0, :, st] = 1.0
    a_log = np.full((ch, st), -30.0, np.float32)
    zero, state, out = B.f32(np.zeros(ch)), B.f32(np.zeros(ch * st)), B.out(n * ch)
    (xs, xv), (ds, _), (bs, _), (zs, zv) = B.act(x), B.act(np.zeros((1, n, ch))), B.act(bc), B.act(np.full((1, n, ch), 2.0))
    dev.selective_scan(xs, ds, bs, zs, B.f32(a_log), zero, zero, state, out, 1, n, ch, st)
    want = np.log(2.0) * xv[0, 0] * Z.silu(2.0)
    assert close(B.read(out, (n, ch)), np.tile(want, (n, 1)), 8e-3 if bf16 else 2e-5)
    assert close(state.to_vec().reshape(ch, st).astype(f64)[:, 0], np.log(2.0) * xv[0, 0], 1e-5)


# ---- mechanisms without an operator: the stream after a layer in which everything else is silent ----
def only(cfg, seed, *keep):
    """Random weights with the output projections of attention, scan and feed-forward zero, but for the names that end in one of
    ``keep``."""
    w = separate_experts(cfg, synth.zidevik_weights(cfg, seed))
    for k, a in w.items():
        if k.endswith((".o", ".down", "side.norm")) and not k.endswith(tuple(keep)):
            w[k] = np.zeros_like(a)
    return w


def stream_err(dev, cfg, w, dtype, t, portion=None, batch=1):
    m = Model.new(cfg, w, dev, batch, max(t, 32), dtype)
    m.set_option("keep_layers", 1)
    rows = synth.tokens(31, (batch, t), cfg.vocab)
    m.prefill(rows, all_logits=True)
    got, worst = m.layer_outputs(), 0.0
    ref = reference(cfg, w)
    for b in range(batch):
        layers = []
        want = ref.fwd(rows[b], ref.new_state(), layers)
        worst = max(worst, float(np.max(np.abs(got[:, b] - np.stack(layers)))) / float(np.max(np.abs(layers))),
                    float(np.max(np.abs(m.prefill_logits()[b] - want)) / np.max(np.abs(want))))
    m.close()
    return worst


ATT, SCAN = (2, 1, 16, 16, 16, 100.0, 0.3), (32, 8, 2, 8)


@pytest.mark.parametrize("dtype,tol", [(DType.F32, 2e-5), (DType.BF16, 2e-2)])
@pytest.mark.parametrize("t,batch", [(2, 1), (40, 1), (300, 2)])
@pytest.mark.parametrize("experts", [Experts(4, 1, 24), Experts(7, 3, 40, 56), Experts(3, 3, 16), Experts(40, 2, 8), Experts(1, 1, 64)])
def test_routed_experts(dev, dtype, tol, t, batch, experts):
    """Groups of many sizes, empty ones among them, one expert for all rows and all experts for each."""
    cfg = Config(vocab=61, width=72, eps=1e-5, layers=[layer(ATT, SCAN, experts)])
    assert stream_err(dev, cfg, only(cfg, 600, ".down"), dtype, t, batch=batch) < tol


@pytest.mark.parametrize("dtype,tol", [(DType.F32, 2e-5), (DType.BF16, 2e-2)])
def test_all_rows_to_one_expert(dev, dtype, tol):
    cfg = Config(vocab=61, width=72, eps=1e-5, layers=[layer(ATT, SCAN, Experts(6, 1, 24))])
    w = only(cfg, 601, ".down")
    w["embed"] = w["embed"].copy()
    w["embed"][:, 0], w["embed"][:, 1:6] = synth.to_bf16_bits(np.float32(3.0)), 0
    assert stream_err(dev, cfg, w, dtype, 200) < tol


@pytest.mark.parametrize("dtype,tol", [(DType.F32, 2e-5), (DType.BF16, 2e-2)])
@pytest.mark.parametrize("ff", [8, 33, 200])
def test_gated_feed_forward(dev, dtype, tol, ff):
    cfg = Config(vocab=61, width=72, eps=1e-5, layers=[layer(ATT, SCAN, ff), layer(ATT, SCAN, ff)])
    assert stream_err(dev, cfg, only(cfg, 602, ".down"), dtype, 70) < tol


@pytest.mark.parametrize("dtype,tol", [(DType.F32, 2e-5), (DType.BF16, 3e-2)])
@pytest.mark.parametrize("dim", [1, 9, 64])
def test_token_input(dev, dtype, tol, dim):
    """Every layer takes its own part of the table, also when it runs twice."""
    cfg = Config(vocab=61, width=72, eps=1e-5, side_dim=dim, loop=Loop(1, 3, 2), layers=[layer(ATT, SCAN, None) for _ in range(4)])
    assert stream_err(dev, cfg, only(cfg, 603, "side.norm"), dtype, 40, batch=2) < tol


@pytest.mark.parametrize("dtype,tol", [(DType.F32, 2e-5), (DType.BF16, 3e-2)])
@pytest.mark.parametrize("start,stop,times", [(0, 1, 1), (0, 3, 2), (2, 3, 4), (1, 2, 3)])
def test_loop_input_and_soft_cap(dev, dtype, tol, start, stop, times):
    cfg = Config(vocab=61, width=72, eps=1e-5, loop=Loop(start, stop, times), logit_softcap=0.7, layers=[layer(ATT, SCAN, None) for _ in range(3)])
    assert stream_err(dev, cfg, only(cfg, 604), dtype, 40) < tol


@pytest.mark.parametrize("dtype,tol", [(DType.F32, 2e-5), (DType.BF16, 3e-2)])
@pytest.mark.parametrize("keep", ["left.o", "right.o"])
def test_either_mixer(dev, dtype, tol, keep):
    cfg = Config(vocab=61, width=72, eps=1e-5, layers=[layer(ATT, SCAN, None, (0.6, 1.7)), layer(ATT, SCAN, None, (1.9, 0.4))])
    assert stream_err(dev, cfg, only(cfg, 605, keep), dtype, 70, batch=2) < tol
