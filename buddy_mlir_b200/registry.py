"""Model registry: named shapes, and model folders (config.json + model.safetensors) whose
architecture is known."""
import json
import os

from . import butolorn, config, talazen

# architecture name in config.json -> parser of that file
ARCHITECTURES = {"Butolorn": butolorn.parse, "Talazen": talazen.parse}

# shapes of the blob-loaded models by name
SHAPES = {c.name: c for c in (config.DEEPSEEK_R1_1P5B, config.QWEN3_8B, config.TINY_QWEN2,
                              config.TINY_QWEN3, config.TINY_MEGA)}


def model_config(folder, dtype="bfloat16", max_len=4096):
    """Configuration of a model folder."""
    with open(os.path.join(folder, "config.json")) as f:
        c = json.load(f)
    name = c.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[name](c, dtype=dtype, max_len=max_len)


def load_model(folder, dtype="bfloat16", max_len=4096):
    """A ModelSession with the folder's weights, ready to run."""
    from .session import ModelSession
    s = ModelSession(model_config(folder, dtype, max_len))
    s.load_safetensors(os.path.join(folder, "model.safetensors"))
    return s
