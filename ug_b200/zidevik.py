"""Zidevik on the layer-list engine: layers in the parallel form."""
from . import hybrid
from .hybrid import CConfig, CLayer, HybridModel
from .zidevik_config import (Attention, Config, Experts, Layer, Loop, Scan, weight_names,  # noqa: F401 (re-exported)
                             weight_shapes)


class Model(HybridModel):
    weight_shapes = staticmethod(weight_shapes)

    @staticmethod
    def describe(cfg):
        cc = CConfig(form=hybrid.FORM_PARALLEL, side_dim=cfg.side_dim, logit_softcap=cfg.logit_softcap)
        if cfg.loop:
            cc.loop_start, cc.loop_stop, cc.loop_times = cfg.loop.start, cfg.loop.stop, cfg.loop.times
        layers = []
        for l in cfg.layers:
            a, s = l.left, l.right
            c = CLayer(mixer=hybrid.MIXER_ATTENTION_SCAN, heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, scale=a.scale,
                       rot_dims=a.rot_dims, rot_interleaved=1, rot_base=a.rot_base, qk_norm=1, attention_scale=l.left_scale,
                       inner=s.inner, state=s.state, conv=s.conv, dt_rank=s.dt_rank, scan_scale=l.right_scale,
                       feed_forward=hybrid.FF_NONE)
            if isinstance(l.mlp, Experts):
                c.feed_forward, c.ff = hybrid.FF_EXPERTS, l.mlp.shared or 0
                c.experts, c.top, c.expert_ff = l.mlp.count, l.mlp.top, l.mlp.ff
            elif l.mlp is not None:
                c.feed_forward, c.ff = hybrid.FF_GATED, l.mlp
            layers.append(c)
        return cc, layers
