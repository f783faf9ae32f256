"""Model registry: the architecture a checkpoint's config.json names -> the class that reads it and builds its archives."""
import json
import os

from . import kernel_call as kc
from .fokonex import FokonexModel
from .zisevik import ZisevikModel

ARCHITECTURES = {m.CONFIG.ARCHITECTURE: m for m in (FokonexModel, ZisevikModel)}
DTYPES = {"bfloat16": kc.DTYPE_BF16, "float32": kc.DTYPE_F32}


def load_model(path, dtype="bfloat16"):
    """The model in folder `path` (config.json, model.safetensors), its matrix products in `dtype`."""
    with open(os.path.join(path, "config.json"), encoding="utf-8") as f:
        name = json.load(f).get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"{path}: unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    if dtype not in DTYPES:
        raise ValueError(f"unknown dtype {dtype!r} (known: {', '.join(DTYPES)})")
    return ARCHITECTURES[name].load(path, DTYPES[dtype])
