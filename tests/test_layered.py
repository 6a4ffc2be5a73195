"""Layered decoders on the CPU: configuration, tensor names, registry, trace protocol, ABI mirrors and host-side checks."""
import ctypes as C
import io
import json
import math

import numpy as np
import pytest

import layered_oracle as lo
from kmll_b200 import lib, pefisun, registry, trace
from kmll_b200 import runtime as rt
from kmll_b200.checkpoint import CheckpointError, write_safetensors

YARN = {"factor": 4.0, "original": 128, "fast": 16.0, "slow": 2.0}


def config(**kw):
    c = {"architecture": "Pefisun", "width": 40, "vocab": 90, "max_positions": 64, "norm": {"eps": 1e-4}, "layers": [
        {"type": "retention", "mixer": {"heads": 3, "dim": 12, "vdim": 8, "decay": [0.5, 0.9, 1.0], "rot": {"base": 500.0, "dims": 8}}, "mlp": None},
        {"type": "latent_attention", "mixer": {"heads": 2, "dim": 6, "rot_dim": 4, "vdim": 10, "kv_rank": 20, "scale": 0.4, "mask": {"size": 7},
                                               "rot": {"base": 900.0, "dims": 4, "scaling": YARN}}, "mlp": {"kind": "dense", "ff": 50}},
        {"type": "lightning", "mixer": {"heads": 1, "dim": 14, "vdim": 18, "decay": [0.99]}, "mlp": {"kind": "dense", "ff": 30}}]}
    c.update(kw)
    return c


def test_configuration_becomes_layer_descriptions():
    cfg = pefisun.layered_config(config(), max_seq_len=50)
    assert (cfg.dim, cfg.vocab_size, cfg.max_seq_len, cfg.position_rows, cfg.norm_offset) == (40, 90, 50, 64, 1.0) and cfg.norm_eps == 1e-4
    r, a, g = cfg.layers
    assert (r.mixer, r.heads, r.dim, r.vdim, r.rot_dim, r.mlp) == (rt.MIXER_LINEAR_ATTENTION, 3, 12, 8, 8, rt.MLP_NONE)
    assert (r.qkv_act, r.gate_act, r.out_norm) == (rt.ACT_NONE, rt.ACT_SILU, rt.OUT_NORM_PER_HEAD) and r.key_scale == pytest.approx(12 ** -0.5)
    assert (a.mixer, a.kv_rank, a.rot_dim, a.window, a.score_scale, a.ff) == (rt.MIXER_LATENT_ATTENTION, 20, 4, 7, 0.4, 50)
    assert a.rotation.magnitude == pytest.approx(0.1 * math.log(4.0) + 1.0)
    assert (g.qkv_act, g.gate_act, g.out_norm, g.key_scale, g.rot_dim) == (rt.ACT_SILU, rt.ACT_SIGMOID, rt.OUT_NORM_JOINT, 1.0, 0)
    assert pefisun.layered_config(config(), max_seq_len=500).max_seq_len == 64  # never more than the learned positions


def test_every_tensor_has_a_place_of_its_shape():
    c = config()
    cfg = pefisun.layered_config(c)
    shapes = lo.tensor_shapes(c)
    names = pefisun.tensor_names(c)
    assert sorted(n for n, _, _ in names) == sorted(shapes)
    for name, layer, tensor in names:
        assert tuple(cfg.tensor_shape(layer, tensor)) == tuple(shapes[name]), name


@pytest.mark.parametrize("dims,base,scaling", [(8, 500.0, None), (64, 1e4, None), (16, 2.5e5, {"factor": 2.0, "original": 512, "fast": 32.0, "slow": 1.0}),
                                               (4, 900.0, YARN), (32, 1e4, {"factor": 1.0, "original": 64, "fast": 8.0, "slow": 8.0}),
                                               (128, 1e6, {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0})])
def test_rotation_frequencies(dims, base, scaling):
    rot = {"dims": dims, "base": base, **({"scaling": scaling} if scaling else {})}
    want, magnitude = lo.rope_inverse_frequencies(rot)
    got = pefisun.rotation(rot)
    np.testing.assert_allclose(got.freqs, want, rtol=1e-14)
    assert got.magnitude == pytest.approx(magnitude, rel=1e-15)


def test_configuration_errors():
    with pytest.raises(CheckpointError):
        pefisun.layered_config(config(layers=[{"type": "pooling", "mixer": {"heads": 1, "dim": 2, "vdim": 2}, "mlp": None}]))
    bad = config()
    bad["layers"][0]["mixer"]["decay"] = [0.5]
    with pytest.raises(CheckpointError):
        pefisun.layered_config(bad)
    bad = config()
    bad["layers"][1]["mixer"]["rot"]["dims"] = 2
    with pytest.raises(CheckpointError):
        pefisun.layered_config(bad)
    bad = config()
    bad["layers"][1]["mlp"]["kind"] = "routed"
    with pytest.raises(CheckpointError):
        pefisun.layered_config(bad)


def test_registry_goes_by_architecture(tmp_path, monkeypatch):
    calls = []
    monkeypatch.setitem(registry.ARCHITECTURES, "Pefisun", lambda d, c, **kw: calls.append((d, c["width"], kw)))
    monkeypatch.setattr(registry, "load_decoder", lambda d, fmt, max_seq_len=None: (("uniform", fmt, max_seq_len), None))
    d = str(tmp_path)
    (tmp_path / "config.json").write_text(json.dumps(config()))
    registry.load_model(d, "float32", 33)
    assert calls == [(d, 40, {"max_seq_len": 33, "compute_f32": True})]
    with pytest.raises(CheckpointError):
        registry.load_model(d, "float16")
    (tmp_path / "config.json").write_text(json.dumps(config(architecture="Unheard")))
    with pytest.raises(CheckpointError):
        registry.load_model(d)
    (tmp_path / "config.json").write_text(json.dumps({"hidden_size": 8}))
    assert registry.load_model(d, max_seq_len=9) == ("uniform", rt.FORMAT_RS_I8, 9)


def test_checkpoint_reader_checks_types_and_shapes(tmp_path):
    c = config()
    T = {n: (np.asarray(a).view(np.uint32) >> 16).astype(np.uint16) for n, a in lo.random_tensors(c, 1).items()}
    write_safetensors(str(tmp_path / "model.safetensors"), T)
    w = pefisun.ModelWeights(str(tmp_path))
    cfg = pefisun.layered_config(c)
    for name, layer, tensor in pefisun.tensor_names(c):
        np.testing.assert_array_equal(w.read(name, "BF16", cfg.tensor_shape(layer, tensor)), T[name])
    with pytest.raises(CheckpointError):
        w.read("head", "BF16", (90, 41))
    with pytest.raises(CheckpointError):
        w.read("head", "F32", (90, 40))


class FakeSession:
    """Records the portions; the logits of a place are (tokens so far, token)."""

    def __init__(self):
        self.seen, self.resets = [], 0

    def reset_sequence(self):
        self.seen, self.resets = [], self.resets + 1

    def extend(self, tokens, want=()):
        assert list(want) == sorted(set(want))
        base = len(self.seen)
        self.seen += list(tokens)
        return np.array([[base + w + 1, tokens[w]] for w in want], dtype=np.float32).reshape(len(want), 2)


def test_trace_replay_protocol(tmp_path):
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [4, 5, 6], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [7], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [9, 8], "want": [1]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": [3], "want": [0]}], "end": ["a"]}]
    out, s = io.StringIO(), FakeSession()
    trace.replay(s, [json.dumps(x) + "\n" for x in steps] + ["\n"], str(tmp_path), out)
    assert out.getvalue().split("\n") == ["done 0", "done 1", "done 2", "done 3", ""]
    got = {n: np.fromfile(tmp_path / f"{n}.f32", "<f4").reshape(-1, 2).tolist() for n in (0, 2, 3)}
    assert got == {0: [[3, 6], [1, 4]], 2: [[2, 8]], 3: [[1, 3]]} and not (tmp_path / "1.f32").exists()
    assert s.resets == 6  # every request begins and ends with an empty sequence
    with pytest.raises(ValueError):
        trace.replay(FakeSession(), [json.dumps({"step": 0, "entries": [{"id": i, "tokens": [1], "want": []} for i in "ab"], "end": []})], str(tmp_path), out)


def test_struct_mirrors_match_the_library():
    handle = lib.load()
    assert handle.kmll_layer_spec_bytes() == C.sizeof(rt._LayerSpec)
    assert handle.kmll_layered_config_bytes() == C.sizeof(rt._LayeredConfig)
    s = rt.LayerSpec(mixer=1, heads=2, dim=3, vdim=4, kv_rank=5, rot_dim=6, window=7, score_scale=0.5, qkv_act=1, gate_act=2, out_norm=1, key_scale=0.25,
                     mlp=1, ff=9, mlp_act=3)._c()
    first = [getattr(s.mixers[0], n) for n, _ in rt._MixerSpec._fields_]
    assert first[:12] == [1, 2, 3, 4, 5, 6, 7, 0.5, 1, 2, 1, 0.25] and (s.mlp, s.ff, s.mlp_act, s.mixers[1].mixer) == (1, 9, 3, rt.MIXER_NONE)
    s = rt.LayerSpec(3, 2, 3, 4, beside=rt.MixerSpec(4, 6, 7, 8, kv_heads=3, chunk=9, head_gate=1, out_scale=0.5, q_scale=0.25, decay_kind=2, decay_tau=4.0,
                                                     decay_rank=10, delta=1, conv=11, unit_eps=0.125, gate_rank=12))._c()
    second = [getattr(s.mixers[1], n) for n, _ in rt._MixerSpec._fields_]
    assert s.mixers[0].mixer == 3 and second[:4] == [4, 6, 7, 8] and second[12:] == [3, 9, 1, 0.5, 0.25, 2, 4.0, 10, 1, 11, 0.125, 12]


@pytest.mark.parametrize("change", [dict(heads=0), dict(rot_dim=3), dict(mixer=7), dict(mixer=rt.MIXER_LINEAR_ATTENTION, rot_dim=8, dim=4), dict(kv_rank=0),
                                    dict(window=-1), dict(mlp=1, ff=0), dict(mlp=5)])
def test_bad_descriptions_are_refused_on_the_host(change):
    spec = dict(mixer=rt.MIXER_LATENT_ATTENTION, heads=2, dim=8, vdim=8, kv_rank=16, rot_dim=4, window=5)
    spec.update(change)
    handle = lib.load()
    cfg = rt.LayeredConfig(dim=32, vocab_size=50, layers=[], max_seq_len=64, position_rows=64)._c()
    cfg.n_layers = 1
    h = C.c_void_p()
    assert handle.kmll_layered_create(C.byref(cfg), C.byref(rt.LayerSpec(**spec)._c()), C.byref(h)) in (-2, -3)
    cfg.max_seq_len = 65  # more positions than learned vectors
    good = rt.LayerSpec(mixer=rt.MIXER_LATENT_ATTENTION, heads=2, dim=8, vdim=8, kv_rank=16, rot_dim=4)._c()
    assert handle.kmll_layered_create(C.byref(cfg), C.byref(good), C.byref(h)) == -2 and b"positions" in handle.kmll_last_error()


# ---- the oracle itself: two evaluations of the same equations -----------------------------------------------------------
def test_oracle_recurrence_equals_its_closed_sum():
    rng = np.random.default_rng(3)
    q, k, v = (rng.standard_normal((2, 9, d)) for d in (5, 5, 4))
    decay = [0.7, 0.95]
    got = lo.linear_recurrence(q, k, v, decay)
    for n in range(2):
        for i in range(9):
            want = sum(decay[n] ** (i - j) * (q[n, i] @ k[n, j]) * v[n, j] for j in range(i + 1))
            np.testing.assert_allclose(got[n, i], want, rtol=1e-12)


def test_oracle_rotation_keeps_distances_and_passes_the_rest():
    rng = np.random.default_rng(4)
    x = rng.standard_normal((6, 10))
    rot = {"dims": 6, "base": 100.0}
    a, b = lo.rotate(x, np.arange(6), rot), lo.rotate(x, np.arange(6) + 11, rot)
    np.testing.assert_allclose(a @ a.T, b @ b.T, atol=1e-12)  # scores depend on distances only
    np.testing.assert_array_equal(a[:, 6:], x[:, 6:])
    np.testing.assert_allclose(a[0], x[0])
    c, s = math.cos(2 * 100.0 ** (-2 / 6)), math.sin(2 * 100.0 ** (-2 / 6))
    np.testing.assert_allclose([a[2, 1], a[2, 4]], [x[2, 1] * c - x[2, 4] * s, x[2, 4] * c + x[2, 1] * s])
