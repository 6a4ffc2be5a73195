"""Model registry: a model directory's config.json names the architecture, the architecture names its loader.  A config.json
without an `architecture` is a text config as kmll reads it (the uniform quantized decoder)."""
from __future__ import annotations

import json
import os

from . import pefisun
from . import runtime as rt
from . import somopel
from .checkpoint import CheckpointError, load_decoder

# architecture -> loader(model_dir, config, max_seq_len, compute_f32)
ARCHITECTURES = {"Pefisun": pefisun.load, "Somopel": somopel.load}


def read_config(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)


def load_model(model_dir: str, dtype: str = "bfloat16", max_seq_len: int | None = None, fmt: int = rt.FORMAT_RS_I8) -> rt.Decoder:
    """A decoder with the directory's weights.  dtype: "bfloat16" (how the model is served) or "float32" (f32 throughout).
    kmll's text models are quantized to `fmt` and compute on f32 activations with either dtype."""
    if dtype not in ("bfloat16", "float32"):
        raise CheckpointError(f"unknown dtype {dtype!r}")
    config = read_config(model_dir)
    name = config.get("architecture")
    if name is None:
        return load_decoder(model_dir, fmt, max_seq_len=max_seq_len)[0]
    if name not in ARCHITECTURES:
        raise CheckpointError(f"unknown architecture {name!r}; known: {', '.join(sorted(ARCHITECTURES))}")
    return ARCHITECTURES[name](model_dir, config, max_seq_len=max_seq_len, compute_f32=dtype == "float32")


__all__ = ["ARCHITECTURES", "load_model", "read_config"]
