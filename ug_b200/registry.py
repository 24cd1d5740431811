"""Model registry: which class runs a model folder (config.json and *.safetensors), decided by its config."""
import glob
import json
import os

from .device import DType, UgError


def _llama(config, st, dev, batch, t_max, dtype):
    from . import llama
    if dtype != DType.BF16:
        raise UgError(6, "the fused Llama engine computes in bf16; ug_b200.llama_graph runs the model in f32")
    cfg = llama.Config.from_dict(config)
    return llama.Model.from_safetensors(cfg, st, dev, batch, min(t_max, cfg.max_position_embeddings))


def _kabidra(config, st, dev, batch, t_max, dtype):
    from . import kabidra
    return kabidra.Model.from_safetensors(kabidra.Config.from_dict(config), st, dev, batch, t_max, dtype)


def _zidevik(config, st, dev, batch, t_max, dtype):
    from . import zidevik
    return zidevik.Model.from_safetensors(zidevik.Config.from_dict(config), st, dev, batch, t_max, dtype)


# architecture name -> loader; precisions each can run in
ARCHITECTURES = {"Llama": _llama, "Kabidra": _kabidra, "Zidevik": _zidevik}
DTYPES = {"Llama": (DType.BF16,), "Kabidra": (DType.BF16, DType.F32), "Zidevik": (DType.BF16, DType.F32)}


def architecture(config):
    """Architecture name of a parsed config.json: its "architecture" entry, or Llama for the Hugging Face layout
    ("architectures" / "model_type", or just the Llama fields)."""
    name = config.get("architecture")
    if name in ARCHITECTURES:
        return name
    if name is None and ("LlamaForCausalLM" in config.get("architectures", ()) or config.get("model_type") == "llama" or
                         "num_key_value_heads" in config):
        return "Llama"
    raise UgError(6, f"no model class for architecture {name or config.get('architectures') or config.get('model_type')!r}")


def read_config(path):
    with open(os.path.join(path, "config.json")) as f:
        return json.load(f)


def weight_files(path):
    files = sorted(glob.glob(os.path.join(path, "*.safetensors")))
    if not files:
        raise UgError(1, f"no .safetensors file in {path}")
    return files


def load(path, dev, batch=1, t_max=2048, dtype=DType.BF16):
    """The model in folder ``path`` on device ``dev``, for ``batch`` sequences of up to ``t_max`` positions."""
    from .safetensors import MmapedSafetensors
    config = read_config(path)
    return ARCHITECTURES[architecture(config)](config, MmapedSafetensors(weight_files(path), dev), dev, batch, t_max, DType(dtype))
