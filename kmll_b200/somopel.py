"""Somopel: a decoder whose config.json lists its layers: grouped chunked attention with a gate per head beside gated linear
attention, or the gated delta rule with a decay per key channel and short convolutions; gated GELU feed-forward, layer norms,
learned positions, a normed embedding and tied logits.  Reads the configuration and the tensor names and builds a
LayeredDecoder; every mechanism lives in the layered runtime with its constants as parameters.  The inner sizes of the low-rank
maps are not in config.json: they are the tensors' own."""
from __future__ import annotations

import json

from . import runtime as rt
from .checkpoint import CheckpointError, ModelWeights, load_layered

UNIT_EPS = 1e-6  # inside the root that makes q and k of the delta rule unit vectors


def _attention(m: dict) -> dict:
    return dict(mixer=rt.MIXER_ATTENTION, heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                score_scale=float(m["scale"]), chunk=int(m["mask"]["size"]), head_gate=1, gate_act=rt.ACT_SIGMOID)


def _gated_linear(m: dict, rank: int) -> dict:
    return dict(mixer=rt.MIXER_GATED_LINEAR, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), q_scale=float(m["dim"]) ** -0.5,
                decay_kind=rt.DECAY_LOGISTIC, decay_tau=float(m["tau"]), decay_rank=rank, gate_act=rt.ACT_SILU, out_norm=rt.OUT_NORM_HEAD_WEIGHTED)


def _delta(m: dict, rank: int, gate_rank: int) -> dict:
    return dict(mixer=rt.MIXER_GATED_LINEAR, heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                q_scale=float(m["dim"]) ** -0.5, decay_kind=rt.DECAY_SOFTPLUS, decay_rank=rank, delta=1, conv=int(m["conv"]), unit_eps=UNIT_EPS,
                gate_rank=gate_rank, gate_act=rt.ACT_SIGMOID, out_norm=rt.OUT_NORM_HEAD_WEIGHTED)


# tensor name below '<layer>.mix.' -> tensor id
_LEFT = {"q": rt.T_WQ, "k": rt.T_WK, "v": rt.T_WV, "g": rt.T_GATE, "o": rt.T_WO}
_RIGHT = {**_LEFT, "norm": rt.T_MIX_NORM, "a1": rt.T_DECAY_DOWN, "a2": rt.T_DECAY_UP, "a2.b": rt.T_DECAY_BIAS}
_DELTA = {"q": rt.T_WQ, "k": rt.T_WK, "v": rt.T_WV, "q.conv": rt.T_Q_CONV, "k.conv": rt.T_K_CONV, "v.conv": rt.T_V_CONV, "b": rt.T_BETA,
          "A_log": rt.T_DECAY_LOG, "norm": rt.T_MIX_NORM, "a1": rt.T_DECAY_DOWN, "a2": rt.T_DECAY_UP, "dt_bias": rt.T_DECAY_BIAS,
          "g1": rt.T_GATE_DOWN, "g2": rt.T_GATE_UP, "o": rt.T_WO}
MIXER_TENSORS = {"parallel": {**{"left." + n: t for n, t in _LEFT.items()}, **{"right." + n: rt.T_BESIDE + t for n, t in _RIGHT.items()}},
                 "channel_delta": _DELTA}
MLP_TENSORS = {"gate": rt.T_W1, "up": rt.T_W3, "down": rt.T_W2}


def layered_config(config: dict, shape_of, max_seq_len: int | None = None, compute_f32: bool = False) -> rt.LayeredConfig:
    """shape_of(tensor name) -> its shape in the checkpoint."""
    layers = []
    for i, layer in enumerate(config["layers"]):
        m, mlp, mix = layer["mixer"], layer.get("mlp"), f"l{i}.mix."
        if layer["type"] == "parallel":
            spec = dict(_attention(m["left"]), out_scale=float(m["left_scale"]),
                        beside=rt.MixerSpec(**_gated_linear(m["right"], int(shape_of(mix + "right.a1")[0])), out_scale=float(m["right_scale"])))
        elif layer["type"] == "channel_delta":
            spec = _delta(m, int(shape_of(mix + "a1")[0]), int(shape_of(mix + "g1")[0]))
        else:
            raise CheckpointError(f"layer {i}: unknown mixer {layer['type']!r}")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise CheckpointError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            spec.update(mlp=rt.MLP_GATED, mlp_act=rt.ACT_GELU_TANH, ff=int(mlp["ff"]))
        layers.append(rt.LayerSpec(**spec))
    positions = int(config["max_positions"])
    return rt.LayeredConfig(dim=int(config["width"]), vocab_size=int(config["vocab"]), layers=layers, position_rows=positions,
                            max_seq_len=min(positions, max_seq_len) if max_seq_len else positions, norm_eps=float(config["norm"]["eps"]),
                            compute_f32=compute_f32, norm=rt.NORM_LAYER, embed_scale=float(config["embedding"]["scale"]), embed_norm=True,
                            logit_scale=float(config["logit_scale"]), tie_output=True)


def tensor_names(config: dict):
    """[(checkpoint name, layer or -1, tensor id)] of every tensor of the model."""
    out = [("embed", -1, rt.T_EMBEDDING), ("pos", -1, rt.T_POSITION)]

    def norm(name, layer, weight, bias):
        out.extend([(name, layer, weight), (name + ".b", layer, bias)])

    norm("embed.norm", -1, rt.T_EMBED_NORM, rt.T_EMBED_NORM_BIAS)
    for i, layer in enumerate(config["layers"]):
        norm(f"l{i}.norm1", i, rt.T_ATTENTION_NORM, rt.T_ATTENTION_NORM_BIAS)
        out += [(f"l{i}.mix.{n}", i, t) for n, t in MIXER_TENSORS[layer["type"]].items()]
        if layer.get("mlp") is not None:
            norm(f"l{i}.norm2", i, rt.T_FFN_NORM, rt.T_FFN_NORM_BIAS)
            out += [(f"l{i}.mlp.{n}", i, t) for n, t in MLP_TENSORS.items()]
    norm("final.norm", -1, rt.T_FINAL_NORM, rt.T_FINAL_NORM_BIAS)
    return out


def load(model_dir: str, config: dict, max_seq_len: int | None = None, compute_f32: bool = False) -> rt.LayeredDecoder:
    weights = ModelWeights(model_dir)
    return load_layered(weights, layered_config(config, weights.shape, max_seq_len, compute_f32), tensor_names(config))


def load_dir(model_dir: str, **kw) -> rt.LayeredDecoder:
    with open(f"{model_dir}/config.json") as f:
        return load(model_dir, json.load(f), **kw)
