"""Somopel on the CPU: configuration, tensor names, registry, host-side checks, and the oracle's mechanisms evaluated a second way."""
import copy
import ctypes as C
import json
import math

import numpy as np
import pytest

import somopel_oracle as so
from kmll_b200 import lib, registry, somopel
from kmll_b200 import runtime as rt
from kmll_b200.checkpoint import CheckpointError, ModelWeights, write_safetensors

RANKS = {"a1": 7, "g1": 9, "right.a1": 3}


def config(**kw):
    c = {"architecture": "Somopel", "width": 40, "vocab": 90, "max_positions": 64, "norm": {"eps": 1e-4}, "embedding": {"scale": 3.0}, "logit_scale": 0.5, "layers": [
        {"type": "parallel", "mixer": {"left": {"heads": 6, "kv_heads": 2, "dim": 5, "vdim": 7, "scale": 0.3, "mask": {"size": 9}}, "left_scale": 0.7,
                                       "right": {"heads": 3, "dim": 4, "vdim": 6, "tau": 5.0}, "right_scale": 1.4}, "mlp": {"kind": "dense", "ff": 50}},
        {"type": "channel_delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 8, "conv": 3}, "mlp": None}]}
    c.update(kw)
    return c


def shape_of(c):
    shapes = so.tensor_shapes(c, RANKS)
    return lambda name: shapes[name]


def test_configuration_becomes_layer_descriptions():
    c = config()
    cfg = somopel.layered_config(c, shape_of(c), max_seq_len=50)
    assert (cfg.dim, cfg.vocab_size, cfg.max_seq_len, cfg.position_rows, cfg.norm, cfg.norm_offset) == (40, 90, 50, 64, rt.NORM_LAYER, 0.0)
    assert (cfg.norm_eps, cfg.embed_scale, cfg.embed_norm, cfg.logit_scale, cfg.tie_output) == (1e-4, 3.0, True, 0.5, True)
    p, d = cfg.layers
    assert (p.mixer, p.heads, p.kv_heads, p.dim, p.vdim, p.chunk, p.score_scale, p.head_gate, p.gate_act, p.out_scale) == \
        (rt.MIXER_ATTENTION, 6, 2, 5, 7, 9, 0.3, 1, rt.ACT_SIGMOID, 0.7)
    r = p.beside
    assert (r.mixer, r.heads, r.dim, r.vdim, r.decay_kind, r.decay_tau, r.decay_rank, r.delta, r.conv, r.unit_eps, r.gate_rank, r.gate_act, r.out_scale) == \
        (rt.MIXER_GATED_LINEAR, 3, 4, 6, rt.DECAY_LOGISTIC, 5.0, 3, 0, 0, 0.0, 0, rt.ACT_SILU, 1.4)
    assert r.q_scale == pytest.approx(0.5) and r.out_norm == rt.OUT_NORM_HEAD_WEIGHTED
    assert (p.mlp, p.mlp_act, p.ff, d.mlp) == (rt.MLP_GATED, rt.ACT_GELU_TANH, 50, rt.MLP_NONE)
    assert (d.mixer, d.heads, d.kv_heads, d.dim, d.vdim, d.decay_kind, d.decay_rank, d.delta, d.conv, d.unit_eps, d.gate_rank, d.gate_act) == \
        (rt.MIXER_GATED_LINEAR, 4, 2, 6, 8, rt.DECAY_SOFTPLUS, 7, 1, 3, 1e-6, 9, rt.ACT_SIGMOID)
    assert d.beside is None and d.q_scale == pytest.approx(6 ** -0.5)
    assert somopel.layered_config(c, shape_of(c), max_seq_len=500).max_seq_len == 64


def test_every_tensor_has_a_place_of_its_shape():
    c = config()
    c["layers"].append({**copy.deepcopy(c["layers"][1]), "mlp": {"kind": "dense", "ff": 12}})
    c["layers"].append({**copy.deepcopy(c["layers"][0]), "mlp": None})
    cfg = somopel.layered_config(c, shape_of(c))
    shapes = so.tensor_shapes(c, RANKS)
    names = somopel.tensor_names(c)
    assert sorted(n for n, _, _ in names) == sorted(shapes) and len({(l, t) for _, l, t in names}) == len(names)
    for name, layer, tensor in names:
        assert tuple(cfg.tensor_shape(layer, tensor)) == tuple(shapes[name]), name
    assert cfg.weight_elements() == sum(int(np.prod(s)) for n, s in shapes.items() if len(s) == 2 and n != "pos")


def test_configuration_errors():
    c = config()
    bad = copy.deepcopy(c)
    bad["layers"][0]["type"] = "serial"
    with pytest.raises(CheckpointError):
        somopel.layered_config(bad, shape_of(c))
    bad = copy.deepcopy(c)
    bad["layers"][0]["mlp"]["kind"] = "routed"
    with pytest.raises(CheckpointError):
        somopel.layered_config(bad, shape_of(c))


def test_registry_and_checkpoint(tmp_path, monkeypatch):
    c = config()
    (tmp_path / "config.json").write_text(json.dumps(c))
    T = {n: (np.asarray(a).view(np.uint32) >> 16).astype(np.uint16) for n, a in so.random_tensors(c, 1, ranks=RANKS).items()}
    write_safetensors(str(tmp_path / "model.safetensors"), T)
    w = ModelWeights(str(tmp_path))
    assert w.shape("l0.mix.right.a1") == (3, 40)
    placed = {}

    class Recorder:
        def __init__(self, cfg):
            self.cfg = cfg

        def set_tensor(self, layer, tensor, values):
            placed[layer, tensor] = values

    monkeypatch.setattr(rt, "LayeredDecoder", Recorder)
    dec = registry.load_model(str(tmp_path), "float32", 33)
    assert dec.cfg.compute_f32 and dec.cfg.max_seq_len == 33 and len(placed) == len(T)
    for name, layer, tensor in somopel.tensor_names(c):
        np.testing.assert_array_equal(placed[layer, tensor], T[name])


GOOD = dict(mixer=rt.MIXER_GATED_LINEAR, heads=4, kv_heads=2, dim=8, vdim=8, decay_kind=rt.DECAY_SOFTPLUS, decay_rank=4, delta=1, conv=4, unit_eps=1e-6, gate_rank=4,
            out_norm=rt.OUT_NORM_HEAD_WEIGHTED)


@pytest.mark.parametrize("change", [dict(kv_heads=3), dict(kv_heads=-1), dict(decay_kind=0), dict(decay_kind=3), dict(decay_kind=rt.DECAY_LOGISTIC, decay_tau=0.0),
                                    dict(decay_rank=0), dict(gate_rank=-1), dict(conv=17), dict(unit_eps=-1.0), dict(rot_dim=4), dict(dim=513),
                                    dict(out_norm=rt.OUT_NORM_JOINT), dict(chunk=-1), dict(mlp=rt.MLP_GATED, ff=4), dict(mlp=rt.MLP_GATED, mlp_act=rt.ACT_SILU, ff=0),
                                    dict(mixer=rt.MIXER_ATTENTION, window=3, chunk=4), dict(mixer=rt.MIXER_ATTENTION, rot_dim=4),
                                    dict(beside=rt.MixerSpec(rt.MIXER_LATENT_ATTENTION, 2, 4, 4, kv_rank=4)), dict(beside=rt.MixerSpec(9, 2, 4, 4))])
def test_bad_descriptions_are_refused_on_the_host(change):
    handle = lib.load()
    cfg = rt.LayeredConfig(dim=32, vocab_size=50, layers=[], max_seq_len=64, position_rows=64)._c()
    cfg.n_layers = 1
    h = C.c_void_p()
    spec = {**GOOD, **change}
    assert handle.kmll_layered_create(C.byref(cfg), C.byref(rt.LayerSpec(**spec)._c()), C.byref(h)) in (-2, -3)
    cfg.norm = 2
    assert handle.kmll_layered_create(C.byref(cfg), C.byref(rt.LayerSpec(**GOOD)._c()), C.byref(h)) == -2


def test_unknown_tensors_are_errors():
    cfg = somopel.layered_config(config(), shape_of(config()))
    with pytest.raises(KeyError):
        cfg.tensor_shape(1, rt.T_DKV)
    with pytest.raises(KeyError):
        cfg.tensor_shape(1, rt.T_BESIDE + rt.T_WQ)


# ---- the oracle itself: second evaluations of the same equations --------------------------------------------------------
def test_oracle_decayed_attention_equals_its_closed_sum():
    rng = np.random.default_rng(3)
    q, k, v = (rng.standard_normal((2, 9, d)) for d in (5, 5, 4))
    alpha = rng.uniform(0.3, 1.0, (2, 9, 5))
    got = so.decayed_linear_attention(q, k, v, alpha)
    for h in range(2):
        for i in range(9):
            want = sum(np.sum(q[h, i] * k[h, j] * np.prod(alpha[h, j + 1:i + 1], axis=0)) * v[h, j] for j in range(i + 1))
            np.testing.assert_allclose(got[h, i], want, rtol=1e-12)


def test_oracle_delta_rule_is_a_triangular_system():
    rng = np.random.default_rng(4)
    H, t, d = 2, 8, 5
    q, k = (so.unit(rng.standard_normal((1, t, d))) for _ in range(2))
    v, g, beta = rng.standard_normal((H, t, 3)), rng.uniform(0.2, 1.0, (H, t, d)), rng.uniform(0, 1, (t, H))
    got = so.delta_rule(q, k, v, g, beta)
    for h in range(H):
        def pair(a, i, j):
            return np.sum(a[0, i] * k[0, j] * np.prod(g[h, j + 1:i + 1], axis=0))
        L = np.array([[beta[i, h] * pair(k, i, j) if j < i else 0.0 for j in range(t)] for i in range(t)])
        U = np.linalg.solve(np.eye(t) + L, beta[:, h:h + 1] * v[h])
        A = np.array([[pair(q, i, j) if j <= i else 0.0 for j in range(t)] for i in range(t)])
        np.testing.assert_allclose(got[h], A @ U, rtol=1e-10)


def test_oracle_delta_rule_overwrites_a_key():
    k = so.unit(np.array([[[1.0, 2.0], [1.0, 2.0]]]))
    v = np.array([[[3.0], [5.0]]])
    out = so.delta_rule(k, k, v, np.ones((1, 2, 2)), np.ones((2, 1)))
    np.testing.assert_allclose(out[0, :, 0], [3.0, 5.0], rtol=1e-5)  # reads back what the token itself wrote


def test_oracle_chunks_and_convolution():
    rng = np.random.default_rng(5)
    q, k, v = rng.standard_normal((2, 10, 4)), rng.standard_normal((1, 10, 4)), rng.standard_normal((1, 10, 3))
    got = so.chunked_attention(q, k, v, 0.7, 4)
    for lo in (0, 4, 8):  # a chunk is a sequence of its own
        hi = min(lo + 4, 10)
        np.testing.assert_allclose(got[:, lo:hi], so.chunked_attention(q[:, lo:hi], k[:, lo:hi], v[:, lo:hi], 0.7, 100))
    np.testing.assert_allclose(got[:, 4], np.repeat(v[:, 4], 2, axis=0))
    x, taps = rng.standard_normal((7, 3)), rng.standard_normal((3, 4))
    y = so.short_convolution(x, taps)
    for t in range(7):
        want = sum(x[t - j] * taps[:, 3 - j] for j in range(4) if t >= j)
        np.testing.assert_allclose(y[t], want)


def test_oracle_scalar_functions():
    z = np.linspace(-30, 30, 61)
    np.testing.assert_allclose(so.softplus(z), [math.log1p(math.exp(-abs(x))) + max(x, 0.0) for x in z])
    np.testing.assert_allclose(np.exp(so.log_sigmoid(z)), so.sigmoid(z), rtol=1e-12)
    x = np.random.default_rng(6).standard_normal((3, 50)) * 4 + 2
    n = so.layer_norm(x, np.ones(50), np.zeros(50), 0.0)
    np.testing.assert_allclose(n.mean(1), 0, atol=1e-12)
    np.testing.assert_allclose(n.std(1), 1)
