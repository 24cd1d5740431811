"""Plain CPU implementation of the Zidevik decoder -- TEST INFRASTRUCTURE ONLY.

numpy in float64, one function per mechanism, one sequence at a time and no
blocking, caching of intermediate products or fusion: every function is the
equation it names.  Nothing here is shared with the product path; the engine
(csrc/hybrid_parallel.cu) is checked against it.

A model is described by the dictionary that config.json holds and by a mapping
tensor name -> float array.  ``Model.fwd`` consumes any number of new tokens of
one sequence and moves that sequence's ``state`` forward.
"""
import numpy as np


# ------------------------------------------------------------- mechanisms ---
def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-np.asarray(x, np.float64)))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


def rms(x, eps):
    """x_i / sqrt(mean_j x_j^2 + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rotate(x, pos, base, dims):
    """Interleaved rotary positions: x [t, heads, dim]; dimensions 2i and 2i + 1 < dims of the row at position p turn by
    p base^(-2i / dims), the others stay."""
    out = x.copy()
    for i in range(dims // 2):
        a = np.asarray(pos, np.float64)[:, None] * base ** (-2.0 * i / dims)
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[:, :, 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def softmax(s):
    e = np.exp(s - np.max(s, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


def grouped_attention(q, k, v, scale, pos0):
    """q [t, H, dim] at positions pos0 .., k / v [pos0 + t, G, dim / vdim]; query head h reads key head h // (H / G) and
    the keys at positions <= its own.  [t, H, vdim]."""
    t, heads, _ = q.shape
    share = heads // k.shape[1]
    out = np.empty((t, heads, v.shape[2]))
    for i in range(t):
        last = pos0 + i + 1
        for h in range(heads):
            w = softmax(k[:last, h // share] @ q[i, h] * scale)
            out[i, h] = w @ v[:last, h // share]
    return out


def causal_conv(h, w, b, past):
    """silu(b + sum_j w[:, j] h_{t - (taps - 1) + j}); ``past``: the taps - 1 rows before h[0].  (result, new past)"""
    taps = w.shape[1]
    full = np.concatenate([past, h], axis=0)
    out = np.zeros_like(h) + b
    for t in range(h.shape[0]):
        for j in range(taps):
            out[t] += w[:, j] * full[t + j]
    return silu(out), full[full.shape[0] - (taps - 1):]


def selective_scan(x, dt, a, b, c, d, state):
    """S <- exp(dt A) S + dt x B, y = S C + D x; x, dt [t, inner], a [inner, N], b, c [t, N], state [inner, N].
    (all y, last S)"""
    out = np.empty_like(x)
    for t in range(x.shape[0]):
        state = np.exp(dt[t][:, None] * a) * state + (dt[t] * x[t])[:, None] * b[t][None, :]
        out[t] = state @ c[t] + d * x[t]
    return out, state


def gated(h, gate, up, down):
    """down(silu(gate h) * (up h))"""
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(z, top):
    """Experts with the ``top`` largest sigmoid scores of one token, best first, and those scores."""
    s = sigmoid(z)
    chosen = np.argsort(-z, kind="stable")[:top]
    return chosen, s[chosen]


def softcap(x, cap):
    return x if not cap else cap * np.tanh(x / cap)


# ------------------------------------------------------------------- model ---
def layer_runs(cfg):
    """(layer, pass entered before it or None) in the order in which layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    lo, hi = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(lo)]
    for t in range(loop["times"]):
        runs += [(i, t if i == lo else None) for i in range(lo, hi)]
    return runs + [(i, None) for i in range(hi, n)]


class Model:
    def __init__(self, cfg, weights):
        self.cfg = cfg
        self.w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
        self.eps = float(cfg["norm"]["eps"])
        self.runs = layer_runs(cfg)

    def new_state(self):
        out = []
        for i, _ in self.runs:
            left, right = (self.cfg["layers"][i]["mixer"][s] for s in ("left", "right"))
            out.append({"k": np.zeros((0, left["kv_heads"], left["dim"])), "v": np.zeros((0, left["kv_heads"], left["vdim"])),
                        "conv": np.zeros((right["conv"] - 1, right["inner"])), "s": np.zeros((right["inner"], right["state"]))})
        return {"pos": 0, "runs": out}

    def _left(self, p, m, h, st, pos0):
        w, t = self.w, len(h)
        pos = pos0 + np.arange(t)
        q = (h @ w[p + "q"].T).reshape(t, m["heads"], m["dim"])
        k = (h @ w[p + "k"].T).reshape(t, m["kv_heads"], m["dim"])
        v = (h @ w[p + "v"].T).reshape(t, m["kv_heads"], m["vdim"])
        q, k = (rms(rotate(a, pos, m["rot"]["base"], m["rot"]["dims"]), self.eps) for a in (q, k))
        st["k"], st["v"] = np.concatenate([st["k"], k]), np.concatenate([st["v"], v])
        return grouped_attention(q, st["k"], st["v"], m["scale"], pos0).reshape(t, -1) @ w[p + "o"].T

    def _right(self, p, m, h, st):
        w, n, r = self.w, m["state"], m["dt_rank"]
        x, z = np.split(h @ w[p + "in"].T, [m["inner"]], axis=1)
        x, st["conv"] = causal_conv(x, w[p + "conv"], w[p + "conv.b"], st["conv"])
        low, b, c = np.split(x @ w[p + "x"].T, [r, r + n], axis=1)
        dt = softplus(low @ w[p + "dt"].T + w[p + "dt.b"])
        y, st["s"] = selective_scan(x, dt, -np.exp(w[p + "A_log"]), b, c, w[p + "D"], st["s"])
        return (y * silu(z)) @ w[p + "o"].T

    def _mlp(self, p, mlp, h):
        w = self.w
        three = lambda q: (w[q + "gate"], w[q + "up"], w[q + "down"])
        if mlp.get("kind", "dense") == "dense":
            return gated(h, *three(p))
        out = np.zeros_like(h)
        z = h @ w[p + "router"].T
        for i in range(len(h)):
            for e, s in zip(*route(z[i], mlp["router"]["top"])):
                out[i] += gated(s * h[i], *three(f"{p}e{e}."))
        if mlp.get("shared"):
            out += gated(h, *three(p + "shared."))
        return out

    def fwd(self, tokens, state, layers_out=None):
        """Logits [len(tokens), vocab] of the next tokens of one sequence; ``layers_out`` (a list) receives the
        residual stream after every layer run."""
        w, cfg, pos0 = self.w, self.cfg, state["pos"]
        tokens = np.asarray(tokens)
        x = x0 = w["embed"][tokens]
        for (i, enter), st in zip(self.runs, state["runs"]):
            p, spec = f"l{i}.", cfg["layers"][i]
            if enter is not None:
                x = np.concatenate([x, x0], axis=1) @ w["loop.in"].T + w["loop.step"][enter]
            h, m = rms(x, self.eps) * w[p + "norm1"], spec["mixer"]
            y = m["left_scale"] * self._left(p + "mix.left.", m["left"], h, st, pos0) + \
                m["right_scale"] * self._right(p + "mix.right.", m["right"], h, st)
            if spec["mlp"] is not None:
                y = y + self._mlp(p + "mlp.", spec["mlp"], h)
            x = x + y
            if cfg.get("token_side"):
                d = cfg["token_side"]["dim"]
                g = gelu_tanh(x @ w[p + "side.gate"].T) * w["side.embed"][tokens][:, i * d:(i + 1) * d]
                x = x + rms(g @ w[p + "side.proj"].T, self.eps) * w[p + "side.norm"]
            if layers_out is not None:
                layers_out.append(x)
        state["pos"] = pos0 + len(tokens)
        return softcap((rms(x, self.eps) * w["final.norm"]) @ w["head"].T, cfg.get("logit_softcap"))
