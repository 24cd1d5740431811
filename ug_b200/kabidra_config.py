"""Kabidra model description: the reader of its config.json, the tensor names in load order and their shapes.
Pure Python: importing this module does not load the CUDA library.

Kabidra is a decoder whose config lists its layers one by one.  Token mixers are a minimal gated recurrent unit or
latent attention without positions; the feed-forward is down(max(up h, 0)^2) or absent.  Every sublayer sits between
two RMS norms and reads its input through a short causal convolution, and a learned average over the embedding and all
layer results so far feeds the next layer.  See include/ugb200.h (ugb_hybrid) for the engine that runs it.
"""
from dataclasses import dataclass
from typing import Optional

MINGRU, LATENT = "mingru", "latent_attention"
_MIXER_FIELDS = {MINGRU: ("width",), LATENT: ("heads", "dim", "vdim", "q_rank", "kv_rank", "scale")}


@dataclass
class Layer:
    type: str
    mixer: dict                  # the sizes _MIXER_FIELDS names for this type
    ff: Optional[int] = None     # feed-forward columns, None = no feed-forward


@dataclass
class Config:
    vocab: int
    width: int
    layers: list
    eps: float
    taps: int                    # of the sublayers' input convolution

    ARCHITECTURE = "Kabidra"

    @staticmethod
    def from_dict(d):
        layers = []
        for i, e in enumerate(d["layers"]):
            kind = e["type"]
            if kind not in _MIXER_FIELDS:
                raise ValueError(f"layer {i}: unknown mixer {kind!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(Layer(kind, {k: e["mixer"][k] for k in _MIXER_FIELDS[kind]}, None if mlp is None else int(mlp["ff"])))
        return Config(vocab=int(d["vocab"]), width=int(d["width"]), layers=layers, eps=float(d["norm"]["eps"]),
                      taps=int(d["canon"]["taps"]))

    @staticmethod
    def from_json(path):
        import json
        with open(path) as f:
            return Config.from_dict(json.load(f))

    def to_dict(self):
        """The config.json this configuration was (or could have been) read from."""
        return {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.eps}, "canon": {"taps": self.taps},
                "layers": [{"type": l.type, "mixer": dict(l.mixer),
                            "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}} for l in self.layers]}

    @staticmethod
    def like_llama_1b(layers=22, vocab=32000):
        """Layers of the size of the 1.1B Llama benchmark model: width 2048, feed-forward 5632, every fourth mixer an
        attention with 16 heads of 128 over a latent of 512, the others recurrent with 2048 channels."""
        att = dict(heads=16, dim=128, vdim=128, q_rank=768, kv_rank=512, scale=128 ** -0.5)
        return Config(vocab=vocab, width=2048, eps=1e-5, taps=4,
                      layers=[Layer(LATENT, dict(att), 5632) if i % 4 == 3 else Layer(MINGRU, {"width": 2048}, 5632)
                              for i in range(layers)])


def weight_shapes(cfg):
    """Tensor name -> shape, in load order."""
    w, out = cfg.width, {"embed": (cfg.vocab, cfg.width), "embed.norm": (cfg.width,)}
    for i, l in enumerate(cfg.layers):
        p, m = f"l{i}.", l.mixer
        out[p + "norm1"], out[p + "norm1b"] = (w,), (w,)
        if l.type == MINGRU:
            n = m["width"]
            out.update({p + "mix.z": (n, w), p + "mix.z.b": (n,), p + "mix.x": (n, w), p + "mix.x.b": (n,),
                        p + "mix.g": (n, w), p + "mix.o": (w, n)})
        else:
            h, q, c = m["heads"], m["q_rank"], m["kv_rank"]
            out.update({p + "mix.dq": (q, w), p + "mix.dq.norm": (q,), p + "mix.uq": (h * m["dim"], q),
                        p + "mix.dkv": (c, w), p + "mix.dkv.norm": (c,), p + "mix.uk": (h * m["dim"], c),
                        p + "mix.uv": (h * m["vdim"], c), p + "mix.g": (h, w), p + "mix.o": (w, h * m["vdim"])})
        out[p + "canon1"] = (w, cfg.taps)
        if l.ff is not None:
            out.update({p + "norm2": (w,), p + "norm2b": (w,), p + "mlp.up": (l.ff, w), p + "mlp.down": (w, l.ff),
                        p + "canon2": (w, cfg.taps)})
        out[p + "dwa"] = (i + 2,)
    out["final.norm"], out["head"] = (w,), (cfg.vocab, w)
    return out


def weight_names(cfg):
    return list(weight_shapes(cfg))
