"""Pefisun: a decoder whose config.json lists its layers (latent attention with a sliding window, retention, lightning
attention; PolyNorm feed-forward, learned positions, norms stored around zero).  Reads the configuration and the tensor names
and builds a LayeredDecoder; every mechanism lives in the layered runtime with its constants as parameters."""
from __future__ import annotations

import json
import math

from . import runtime as rt
from .checkpoint import CheckpointError, ModelWeights, YarnRopeConfig, load_layered


def inverse_frequencies(dims: int, base: float, yarn: YarnRopeConfig | None = None):
    """Rotary frequencies base^(-2i / dims), i < dims / 2, in float64.  With YaRN the frequencies whose wavelength exceeds the
    original context are divided by the factor, with a linear ramp between the two correction dimensions."""
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if yarn is None:
        return freqs

    def correction(rotations):
        return dims * math.log(yarn.original_max_position_embeddings / (2.0 * math.pi * rotations)) / (2.0 * math.log(base))

    low = max(math.floor(correction(yarn.beta_fast)), 0)
    high = min(math.ceil(correction(yarn.beta_slow)), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        out.append(f / yarn.factor * ramp + f * (1.0 - ramp))
    return out


def rotation(cfg: dict) -> rt.Rotation:
    """A `rot` object: dims, base, optional YaRN `scaling` (its magnitude 0.1 ln(factor) + 1 goes on cos and sin)."""
    s = cfg.get("scaling")
    if s is None:
        return rt.Rotation(inverse_frequencies(int(cfg["dims"]), float(cfg["base"])))
    magnitude = 0.1 * math.log(float(s["factor"])) + 1.0
    yarn = YarnRopeConfig(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"]), magnitude)
    return rt.Rotation(inverse_frequencies(int(cfg["dims"]), float(cfg["base"]), yarn), magnitude)


def _latent_attention(m: dict) -> dict:
    out = dict(mixer=rt.MIXER_LATENT_ATTENTION, kv_rank=int(m["kv_rank"]), rot_dim=int(m["rot_dim"]), score_scale=float(m["scale"]),
               window=int(m["mask"]["size"]) if m.get("mask") else 0)
    if out["rot_dim"]:
        out["rotation"] = rotation(m["rot"])
        if 2 * len(out["rotation"].freqs) != out["rot_dim"]:
            raise CheckpointError(f"latent attention rotates its whole rot_dim part: rot.dims {m['rot']['dims']}, rot_dim {out['rot_dim']}")
    return out


def _retention(m: dict) -> dict:
    out = dict(mixer=rt.MIXER_LINEAR_ATTENTION, qkv_act=rt.ACT_NONE, gate_act=rt.ACT_SILU, out_norm=rt.OUT_NORM_PER_HEAD,
               key_scale=float(m["dim"]) ** -0.5, decay=[float(x) for x in m["decay"]])
    if m.get("rot"):
        out["rotation"] = rotation(m["rot"])
        out["rot_dim"] = 2 * len(out["rotation"].freqs)
    return out


def _lightning(m: dict) -> dict:
    return dict(mixer=rt.MIXER_LINEAR_ATTENTION, qkv_act=rt.ACT_SILU, gate_act=rt.ACT_SIGMOID, out_norm=rt.OUT_NORM_JOINT, key_scale=1.0,
                decay=[float(x) for x in m["decay"]])


# mixer type -> (description from its config, {tensor name below '<layer>.mix.': tensor id})
_LINEAR_TENSORS = {"q": rt.T_WQ, "k": rt.T_WK, "v": rt.T_WV, "g": rt.T_GATE, "o": rt.T_WO}
MIXERS = {
    "latent_attention": (_latent_attention, {"q": rt.T_WQ, "dkv": rt.T_DKV, "dkv.norm": rt.T_DKV_NORM, "uk": rt.T_UK, "uv": rt.T_UV, "o": rt.T_WO}),
    "retention": (_retention, _LINEAR_TENSORS),
    "lightning": (_lightning, {**_LINEAR_TENSORS, "norm": rt.T_MIX_NORM}),
}
MLP_TENSORS = {"up": rt.T_W3, "down": rt.T_W2, "act": rt.T_ACT}


def layered_config(config: dict, max_seq_len: int | None = None, compute_f32: bool = False) -> rt.LayeredConfig:
    layers = []
    for i, layer in enumerate(config["layers"]):
        if layer["type"] not in MIXERS:
            raise CheckpointError(f"layer {i}: unknown mixer {layer['type']!r}")
        m, mlp = layer["mixer"], layer.get("mlp")
        spec = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), **MIXERS[layer["type"]][0](m))
        if "decay" in spec and len(spec["decay"]) != spec["heads"]:
            raise CheckpointError(f"layer {i}: {len(spec['decay'])} decays for {spec['heads']} heads")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise CheckpointError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            spec.update(mlp=rt.MLP_POLYNORM, ff=int(mlp["ff"]))
        layers.append(rt.LayerSpec(**spec))
    positions = int(config["max_positions"])
    return rt.LayeredConfig(dim=int(config["width"]), vocab_size=int(config["vocab"]), layers=layers, position_rows=positions,
                            max_seq_len=min(positions, max_seq_len) if max_seq_len else positions, norm_eps=float(config["norm"]["eps"]), norm_offset=1.0,
                            compute_f32=compute_f32)


def tensor_names(config: dict):
    """[(checkpoint name, layer or -1, tensor id)] of every tensor of the model."""
    out = [("embed", -1, rt.T_EMBEDDING), ("pos", -1, rt.T_POSITION), ("final.norm", -1, rt.T_FINAL_NORM), ("head", -1, rt.T_OUTPUT)]
    for i, layer in enumerate(config["layers"]):
        out.append((f"l{i}.norm1", i, rt.T_ATTENTION_NORM))
        out += [(f"l{i}.mix.{n}", i, t) for n, t in MIXERS[layer["type"]][1].items()]
        if layer.get("mlp") is not None:
            out.append((f"l{i}.norm2", i, rt.T_FFN_NORM))
            out += [(f"l{i}.mlp.{n}", i, t) for n, t in MLP_TENSORS.items()]
    return out


def load(model_dir: str, config: dict, max_seq_len: int | None = None, compute_f32: bool = False) -> rt.LayeredDecoder:
    return load_layered(ModelWeights(model_dir), layered_config(config, max_seq_len, compute_f32), tensor_names(config))


def load_dir(model_dir: str, **kw) -> rt.LayeredDecoder:
    with open(f"{model_dir}/config.json") as f:
        return load(model_dir, json.load(f), **kw)
