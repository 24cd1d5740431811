"""Kabidra on the layer-list engine: layers in the sandwich form."""
from . import hybrid
from .hybrid import CConfig, CLayer, HybridModel
from .kabidra_config import LATENT, MINGRU, Config, Layer, weight_names, weight_shapes  # noqa: F401 (re-exported)

_MIXERS = {MINGRU: hybrid.MIXER_MINGRU, LATENT: hybrid.MIXER_LATENT_ATTENTION}


class Model(HybridModel):
    weight_shapes = staticmethod(weight_shapes)

    @staticmethod
    def describe(cfg):
        cc = CConfig(conv_taps=cfg.taps, depth_average=1, gain_offset=1.0, form=hybrid.FORM_SANDWICH)
        return cc, [CLayer(mixer=_MIXERS[l.type], feed_forward=hybrid.FF_NONE if l.ff is None else hybrid.FF_RELU2, ff=l.ff or 0,
                           **l.mixer) for l in cfg.layers]
