"""Model folders: ``config.json`` and ``model.safetensors``."""
from __future__ import annotations

import json
import os


def read_config(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)


def read_tensors(model_dir: str) -> dict:
    """Name -> tensor on the CPU, in the file's own dtypes."""
    from safetensors.torch import load_file
    return load_file(os.path.join(model_dir, "model.safetensors"))
