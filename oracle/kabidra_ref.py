"""Plain CPU implementation of the Kabidra decoder -- TEST INFRASTRUCTURE ONLY.

numpy in float64, one function per mechanism, one sequence at a time and no
blocking, caching of intermediate products or fusion: every function is the
equation it names.  Nothing here is shared with the product path; the engine
(csrc/hybrid_engine.cu) is checked against it.

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


def rms(x, eps):
    """x_i / sqrt(mean_j x_j^2 + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_centred(x, w, eps):
    """RMS norm whose gain is stored as its distance from one."""
    return rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


def causal_conv(h, w, past):
    """Depthwise causal convolution over time: c_t[i] = sum_j w[i, j] h_{t - (taps - 1) + j}[i].

    ``past`` holds the taps - 1 rows before h[0] (zeros at the start of a sequence).  Returns (c, new past)."""
    taps = w.shape[1]
    full = np.concatenate([past, h], axis=0)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(taps):
            out[t] += w[:, j] * full[t + j]
    return out, full[full.shape[0] - (taps - 1):]


def min_gru(z, candidate, state):
    """S_t = (1 - z_t) S_{t-1} + z_t c_t, element by element.  Returns (all S_t, last S)."""
    out = np.empty_like(z)
    for t in range(z.shape[0]):
        state = (1.0 - z[t]) * state + z[t] * candidate[t]
        out[t] = state
    return out, state


def gru_candidate(u):
    """u + 1/2 on the non-negative side, sigmoid(u) on the negative side (continuous and positive)."""
    return np.where(u >= 0, u + 0.5, sigmoid(u))


def softmax(s):
    e = np.exp(s - np.max(s, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


def latent_attention(q, c, w_uk, w_uv, scale, pos0, heads):
    """q [t, heads, dim] at positions pos0 .., latents c [pos0 + t, rank]; returns [t, heads, vdim].

    Keys and values of head h are rows h * dim .. (h + 1) * dim of w_uk c_j and h * vdim .. of w_uv c_j; query i
    sees j <= pos0 + i."""
    t, _, dim = q.shape
    n = c.shape[0]
    k = (c @ w_uk.T).reshape(n, heads, dim)
    v = (c @ w_uv.T).reshape(n, heads, -1)
    out = np.empty((t, heads, v.shape[2]))
    for i in range(t):
        last = pos0 + i + 1
        for h in range(heads):
            s = (k[:last, h] @ q[i, h]) * scale
            out[i, h] = softmax(s) @ v[:last, h]
    return out


def relu_squared(x):
    return np.square(np.maximum(x, 0.0))


def depth_average(coef, outputs):
    """sum_j coef[j] outputs[j] over the embedding output and every layer result so far."""
    acc = np.zeros_like(outputs[0])
    for a, x in zip(coef, outputs):
        acc = acc + a * x
    return acc


# ------------------------------------------------------------------- model ---
class Model:
    def __init__(self, cfg, weights):
        self.cfg = cfg
        self.w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
        self.eps = float(cfg["norm"]["eps"])
        self.taps = int(cfg["canon"]["taps"])

    def new_state(self):
        width = self.cfg["width"]
        layers = []
        for spec in self.cfg["layers"]:
            st = {"canon1": np.zeros((self.taps - 1, width)), "canon2": np.zeros((self.taps - 1, width))}
            if spec["type"] == "mingru":
                st["s"] = np.zeros(spec["mixer"]["width"])
            else:
                st["c"] = np.zeros((0, spec["mixer"]["kv_rank"]))
            layers.append(st)
        return {"pos": 0, "layers": layers}

    def _mixer(self, i, spec, h, st, pos0):
        p, w, m = f"l{i}.mix.", self.w, spec["mixer"]
        if spec["type"] == "mingru":
            z = sigmoid(h @ w[p + "z"].T + w[p + "z.b"])
            u = h @ w[p + "x"].T + w[p + "x.b"]
            s, st["s"] = min_gru(z, gru_candidate(u), st["s"])
            return (s * silu(h @ w[p + "g"].T)) @ w[p + "o"].T
        if spec["type"] != "latent_attention":
            raise ValueError(spec["type"])
        heads = m["heads"]
        q = norm_plain(h @ w[p + "dq"].T, w[p + "dq.norm"], self.eps) @ w[p + "uq"].T
        c = norm_plain(h @ w[p + "dkv"].T, w[p + "dkv.norm"], self.eps)
        st["c"] = np.concatenate([st["c"], c], axis=0)
        o = latent_attention(q.reshape(len(h), heads, m["dim"]), st["c"], w[p + "uk"], w[p + "uv"], m["scale"], pos0, heads)
        o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
        return o.reshape(len(h), -1) @ w[p + "o"].T

    def fwd(self, tokens, state, layers_out=None):
        """Logits [len(tokens), vocab] of the next tokens of one sequence; ``layers_out`` (a list) receives the
        residual stream after every layer."""
        w, eps, pos0 = self.w, self.eps, state["pos"]
        x = norm_centred(w["embed"][np.asarray(tokens)], w["embed.norm"], eps)
        depth = [x]
        for i, spec in enumerate(self.cfg["layers"]):
            st, p = state["layers"][i], f"l{i}."
            h = norm_centred(x, w[p + "norm1"], eps)
            c, st["canon1"] = causal_conv(h, w[p + "canon1"], st["canon1"])
            x = x + norm_centred(self._mixer(i, spec, h + c, st, pos0), w[p + "norm1b"], eps)
            if spec["mlp"] is not None:
                h = norm_centred(x, w[p + "norm2"], eps)
                c, st["canon2"] = causal_conv(h, w[p + "canon2"], st["canon2"])
                y = relu_squared((h + c) @ w[p + "mlp.up"].T) @ w[p + "mlp.down"].T
                x = x + norm_centred(y, w[p + "norm2b"], eps)
            depth.append(x)
            x = depth_average(w[p + "dwa"], depth)
            if layers_out is not None:
                layers_out.append(x)
        state["pos"] = pos0 + len(tokens)
        return norm_centred(x, w["final.norm"], eps) @ w["head"].T
