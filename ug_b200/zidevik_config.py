"""Zidevik model description: the reader of its config.json, the tensor names in load order and their shapes.
Pure Python: importing this module does not load the CUDA library.

Zidevik is a decoder whose config lists its layers one by one.  A layer's mixer is grouped-query attention with rotary
positions and a selective scan side by side; mixer and feed-forward (gated, or a mixture of gated experts beside a shared
one, or none) read the same norm and are added together; a per-layer input of the token follows.  A stretch of layers runs
several times with the same weights.  See include/ugb200.h (ugb_hybrid, parallel form) for the engine that runs it.
"""
from dataclasses import dataclass
from typing import Optional

PARALLEL = "parallel"


@dataclass
class Attention:                 # left
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot_dims: int
    rot_base: float
    scale: float


@dataclass
class Scan:                      # right
    inner: int
    state: int
    conv: int
    dt_rank: int


@dataclass
class Experts:
    count: int
    top: int
    ff: int
    shared: Optional[int] = None     # columns of the expert every token uses, None = none


@dataclass
class Layer:
    left: Attention
    right: Scan
    left_scale: float
    right_scale: float
    mlp: object = None           # None, an int (columns of a dense feed-forward) or Experts


@dataclass
class Loop:
    start: int
    stop: int
    times: int


@dataclass
class Config:
    vocab: int
    width: int
    layers: list
    eps: float
    loop: Optional[Loop] = None
    side_dim: int = 0            # columns of a layer's token input, 0 = none
    logit_softcap: float = 0.0   # 0 = none

    ARCHITECTURE = "Zidevik"

    @staticmethod
    def from_dict(d):
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] != PARALLEL:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            m = e["mixer"]
            a, s = m["left"], m["right"]
            rot = a.get("rot") or {"dims": 0, "base": 1.0}
            layers.append(Layer(
                Attention(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), int(rot["dims"]), float(rot["base"]), float(a["scale"])),
                Scan(int(s["inner"]), int(s["state"]), int(s["conv"]), int(s["dt_rank"])),
                float(m["left_scale"]), float(m["right_scale"]), _read_mlp(i, e.get("mlp"))))
        loop, side = d.get("loop"), d.get("token_side")
        return Config(vocab=int(d["vocab"]), width=int(d["width"]), layers=layers, eps=float(d["norm"]["eps"]),
                      loop=None if not loop else Loop(int(loop["start"]), int(loop["stop"]), int(loop["times"])),
                      side_dim=0 if not side else int(side["dim"]), logit_softcap=float(d.get("logit_softcap") or 0.0))

    @staticmethod
    def from_json(path):
        import json
        with open(path) as f:
            return Config.from_dict(json.load(f))

    def to_dict(self):
        """The config.json this configuration was (or could have been) read from."""
        out = {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": []}
        for l in self.layers:
            a, s = l.left, l.right
            left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                    "rot": {"dims": a.rot_dims, "base": a.rot_base}}
            right = {"inner": s.inner, "state": s.state, "conv": s.conv, "dt_rank": s.dt_rank}
            out["layers"].append({"type": PARALLEL, "mlp": _write_mlp(l.mlp),
                                  "mixer": {"left": left, "right": right, "left_scale": l.left_scale, "right_scale": l.right_scale}})
        if self.loop:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        return out

    @staticmethod
    def like_llama(width=2048, layers=22, head=64, kv_heads=4, ff=5632, vocab=32000):
        """Layers of the size of a Llama benchmark model (the 1.1B one by default): as many heads as the width holds, a scan of
        twice the width with 16 states; every other feed-forward dense, the others 16 experts of a quarter of its columns, of
        which a token uses 2, beside a shared one of half.  A quarter of the layers, from the third eighth on, runs twice."""
        left = Attention(heads=width // head, kv_heads=kv_heads, dim=head, vdim=head, rot_dims=head, rot_base=10000.0, scale=head ** -0.5)
        right = Scan(inner=2 * width, state=16, conv=4, dt_rank=width // 16)
        lo = 3 * layers // 8
        return Config(vocab=vocab, width=width, eps=1e-5, loop=Loop(lo, lo + max(1, (layers + 2) // 4), 2), side_dim=256, logit_softcap=30.0,
                      layers=[Layer(left, right, 1.0, 1.0, ff if i % 2 == 0 else Experts(16, 2, ff // 4, ff // 2)) for i in range(layers)])


def _read_mlp(i, mlp):
    if mlp is None:
        return None
    kind = mlp.get("kind", "dense")
    if kind == "dense":
        return int(mlp["ff"])
    if kind != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {kind!r}")
    shared = mlp.get("shared")
    return Experts(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]), None if not shared else int(shared["ff"]))


def _write_mlp(mlp):
    if mlp is None:
        return None
    if not isinstance(mlp, Experts):
        return {"kind": "dense", "ff": mlp}
    out = {"kind": "moe", "router": {"experts": mlp.count, "top": mlp.top}, "expert": {"ff": mlp.ff}}
    if mlp.shared:
        out["shared"] = {"ff": mlp.shared}
    return out


def weight_shapes(cfg):
    """Tensor name -> shape, in load order."""
    w, out = cfg.width, {"embed": (cfg.vocab, cfg.width)}
    gated = lambda p, ff: {p + "gate": (ff, w), p + "up": (ff, w), p + "down": (w, ff)}
    if cfg.loop:
        out["loop.in"], out["loop.step"] = (w, 2 * w), (cfg.loop.times, w)
    if cfg.side_dim:
        out["side.embed"] = (cfg.vocab, len(cfg.layers) * cfg.side_dim)
    for i, l in enumerate(cfg.layers):
        p, a, s = f"l{i}.", l.left, l.right
        out[p + "norm1"] = (w,)
        q = p + "mix.left."
        out.update({q + "q": (a.heads * a.dim, w), q + "k": (a.kv_heads * a.dim, w), q + "v": (a.kv_heads * a.vdim, w),
                    q + "o": (w, a.heads * a.vdim)})
        q = p + "mix.right."
        out.update({q + "in": (2 * s.inner, w), q + "conv": (s.inner, s.conv), q + "conv.b": (s.inner,),
                    q + "x": (s.dt_rank + 2 * s.state, s.inner), q + "dt": (s.inner, s.dt_rank), q + "dt.b": (s.inner,),
                    q + "A_log": (s.inner, s.state), q + "D": (s.inner,), q + "o": (w, s.inner)})
        q = p + "mlp."
        if isinstance(l.mlp, Experts):
            out[q + "router"] = (l.mlp.count, w)
            for e in range(l.mlp.count):
                out.update(gated(f"{q}e{e}.", l.mlp.ff))
            if l.mlp.shared:
                out.update(gated(q + "shared.", l.mlp.shared))
        elif l.mlp is not None:
            out.update(gated(q, l.mlp))
        if cfg.side_dim:
            out.update({p + "side.gate": (cfg.side_dim, w), p + "side.proj": (w, cfg.side_dim), p + "side.norm": (w,)})
    out["final.norm"], out["head"] = (w,), (cfg.vocab, w)
    return out


def weight_names(cfg):
    return list(weight_shapes(cfg))
