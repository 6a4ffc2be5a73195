"""Layered decoders on the GPU against the plain restatement in layered_oracle.py: every mechanism alone, prompts, portions,
decoding, window and chunk edges, far keys, odd sizes, re-used sequences, and generation through the session layer."""
import copy
import json

import numpy as np
import pytest

import layered_oracle as lo
from kmll_b200 import pefisun, registry
from kmll_b200 import runtime as rt
from kmll_b200.checkpoint import write_safetensors
from kmll_b200.lib import KmllError, load
from kmll_b200.session import GenerationOptions, SamplingOptions, Session

pytestmark = pytest.mark.gpu

# relative to the root mean square of the logits (or of the residual stream), per position; bf16: activations of the projections
TOL = {"float32": 3e-5, "bfloat16": 4e-2}
DTYPES = ["float32", "bfloat16"]


def retention(heads=2, dim=16, vdim=24, decay=None, rot=None, base=400.0):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [0.93 + 0.06 * i / heads for i in range(heads)],
                                           "rot": {"base": base, "dims": dim if rot is None else rot}}, "mlp": None}


def lightning(heads=2, dim=24, vdim=16, decay=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [0.8 + 0.19 * i / heads for i in range(heads)]},
            "mlp": None}


def latent(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, window=11, scale=0.2, scaling=None, base=3000.0):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = scaling
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                                                  "mask": {"size": window}, "rot": rot}, "mlp": None}


def with_mlp(layer, ff):
    return {**layer, "mlp": {"kind": "dense", "ff": ff}}


def config(layers, width=72, vocab=130, positions=512, eps=1e-5):
    return {"architecture": "Pefisun", "width": width, "vocab": vocab, "max_positions": positions, "norm": {"eps": eps}, "layers": copy.deepcopy(layers)}


YARN = {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}
MIXED = [with_mlp(lightning(), 100), with_mlp(latent(scaling=YARN), 88), with_mlp(retention(rot=8), 120), latent(heads=2, window=70), with_mlp(lightning(3, 8, 40), 56)]


class Model:
    def __init__(self, cfg, dtype, seed=0, tensors=None, max_seq_len=None):
        self.cfg, self.dtype = cfg, dtype
        self.tensors = lo.random_tensors(cfg, seed) if tensors is None else {n: lo.bf16_round(a) for n, a in tensors.items()}
        layered = pefisun.layered_config(cfg, max_seq_len, dtype == "float32")
        self.dec = rt.LayeredDecoder(layered)
        for name, layer, tensor in pefisun.tensor_names(cfg):
            bits = (np.ascontiguousarray(self.tensors[name], dtype=np.float32).view(np.uint32) >> 16).astype(np.uint16)
            self.dec.set_tensor(layer, tensor, bits)

    def tokens(self, n, seed=1):
        return np.random.default_rng(seed).integers(0, self.cfg["vocab"], n)

    def run(self, tokens, portions=None):
        """Logits of every position, the sequence cut into `portions`."""
        self.dec.reset()
        out, at = [], 0
        for n in portions or [len(tokens)]:
            out.append(self.dec.extend(tokens[at:at + n], range(n)))
            at += n
        assert at == len(tokens) and self.dec.position == at
        return np.concatenate(out)

    def oracle(self, tokens, **kw):
        return lo.forward(self.cfg, self.tensors, tokens, **kw)

    def close(self):
        self.dec.close()


def rel(got, want):
    d = got - want
    d = d - d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / np.sqrt((want * want).mean())


def check(got, want, dtype, factor=1.0):
    e = rel(np.asarray(got, dtype=np.float64), want)
    assert np.all(np.isfinite(e)) and e.max() <= factor * TOL[dtype], (int(e.argmax()), float(e.max()))


def parts(n, sizes):
    out = []
    while sum(out) < n:
        out.append(min(sizes[len(out) % len(sizes)], n - sum(out)))
    return out


# ---- mechanisms alone ------------------------------------------------------------------------------------------------------
ALONE = {"retention": retention(), "retention_partial_rotation": retention(3, 20, 12, rot=12), "retention_no_decay": retention(1, 32, 32, decay=[1.0]),
         "retention_fast_decay": retention(2, 16, 16, decay=[0.4, 0.7]), "lightning_fast_decay": lightning(2, 16, 16, decay=[0.0, 0.05]),
         "lightning": lightning(), "lightning_one_head": lightning(1, 40, 8, decay=[0.999]),
         "latent": latent(), "latent_yarn": latent(scaling=YARN), "latent_window_1": latent(window=1), "latent_no_cut": latent(window=512),
         "latent_many_heads": latent(heads=19, dim=8, rot_dim=4, vdim=8, kv_rank=24)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mixer_alone(cuda, name, dtype):
    m = Model(config([ALONE[name]]), dtype, seed=5)
    tokens = m.tokens(90)
    want = m.oracle(tokens)
    check(m.run(tokens), want, dtype)
    check(m.run(tokens[:40], [1] * 40), want[:40], dtype)  # from the first token on, one by one
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_feed_forward_norms_and_positions_alone(cuda, dtype):
    cfg = config([with_mlp(lightning(1, 8, 8), 200)], width=64, eps=3e-3)  # eps large enough to be seen
    T = lo.random_tensors(cfg, 2)
    T["l0.mix.o"] = np.zeros_like(T["l0.mix.o"])  # the mixer adds nothing
    T["l0.mlp.act"] = np.array([0.3, -0.8, 0.6, 0.4])
    T["embed"] = T["embed"] * 0.1
    m = Model(cfg, dtype, tensors=T)
    tokens = m.tokens(20)
    per = []
    want = m.oracle(tokens, per_layer=per)
    check(m.run(tokens), want, dtype)
    check(m.run(tokens, [1] * 20), want, dtype)
    m.dec.reset()
    got = m.dec.layer_residuals(tokens)
    check(got[0], per[0], dtype)
    for changed in ("pos", "l0.norm2", "final.norm"):  # each of them shows
        T2 = {**m.tensors, changed: np.zeros_like(m.tensors[changed])}
        assert rel(lo.forward(cfg, T2, tokens), want).max() > 3 * TOL["bfloat16"], changed
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_stream_layer_by_layer(cuda, dtype):
    m = Model(config(MIXED), dtype, seed=3)
    tokens = m.tokens(75)
    per = []
    m.oracle(tokens, per_layer=per)
    m.dec.reset()
    first = m.dec.layer_residuals(tokens[:33])
    rest = m.dec.layer_residuals(tokens[33:])
    for l, want in enumerate(per):
        check(np.concatenate([first[l], rest[l]]), want, dtype)
    m.close()


# ---- prompts, portions, decoding ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[200], [2], [3, 64, 1, 5], [63, 2, 65], [64], [70, 1, 1, 2], [199, 1]])
def test_cuts_do_not_matter(cuda, dtype, sizes):
    m = Model(config(MIXED), dtype, seed=7)
    tokens = m.tokens(200)
    want = m.oracle(tokens)
    check(m.run(tokens, parts(200, sizes)), want, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_and_first_tokens(cuda, dtype):
    m = Model(config(MIXED), dtype, seed=8)
    tokens = m.tokens(330)
    want = m.oracle(tokens)
    check(m.run(tokens, [5] + [1] * 325), want, dtype)
    for n in (1, 2, 3):
        check(m.run(tokens[:n]), want[:n], dtype)
        check(m.run(tokens[:n], [1] * n), want[:n], dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_sequence_leaves_nothing_behind(cuda, dtype):
    m = Model(config(MIXED), dtype, seed=9)
    a, b = m.tokens(150, 2), m.tokens(37, 3)
    alone = {}
    for name, t in (("a", a), ("b", b)):
        fresh = Model(config(MIXED), dtype, tensors=m.tensors)
        alone[name] = fresh.run(t, parts(len(t), [20, 1]))
        fresh.close()
    for _ in range(2):
        np.testing.assert_array_equal(m.run(a, parts(150, [20, 1])), alone["a"])
        np.testing.assert_array_equal(m.run(b, parts(37, [20, 1])), alone["b"])
    m.close()


def test_prompt_longer_than_one_pass(cuda):
    cfg = config([with_mlp(retention(1, 16, 16), 32), latent(heads=1, window=300), lightning(1, 16, 16, decay=[0.9995])], width=32, vocab=64, positions=4600)
    m = Model(cfg, "bfloat16", seed=4)
    tokens = m.tokens(4400)
    whole = m.run(tokens)
    cut = m.run(tokens, parts(4400, [997, 64, 1]))
    check(cut, whole.astype(np.float64), "bfloat16")
    m.close()


# ---- other sizes ---------------------------------------------------------------------------------------------------------------
ODD = {"odd": (config([with_mlp(retention(3, 10, 7, rot=6), 37), with_mlp(latent(heads=5, dim=9, rot_dim=6, vdim=11, kv_rank=21, window=5), 51),
                       with_mlp(lightning(1, 13, 5), 29)], width=51, vocab=77), 140),
       "ones": (config([with_mlp(retention(1, 2, 1, rot=2), 1), with_mlp(latent(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1, window=2), 3),
                        with_mlp(lightning(1, 1, 1), 2)], width=9, vocab=5), 70),
       "wide_heads": (config([retention(1, 200, 130, rot=64), latent(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=512, window=90),
                              lightning(2, 128, 72)], width=256), 150),
       "long_keys": (config([retention(1, 256, 64), lightning(1, 250, 33)], width=64), 130),
       "beyond_the_fast_forms": (config([retention(1, 300, 16, rot=300), latent(heads=2, dim=200, rot_dim=72, vdim=140, kv_rank=530, window=33)], width=64), 80)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ODD))
def test_other_sizes(cuda, name, dtype):
    cfg, n = ODD[name]
    m = Model(cfg, dtype, seed=11)
    tokens = m.tokens(n)
    want = m.oracle(tokens)
    # (one-wide layers put a root mean square over a single value on everything: rounding is not averaged there)
    factor = 3.0 if name == "ones" else 1.5
    check(m.run(tokens), want, dtype, factor)
    check(m.run(tokens, parts(n, [31, 2, 1, 1])), want, dtype, factor)
    m.close()


# ---- one key that stands out ---------------------------------------------------------------------------------------------------
MARK, ASK = 1, 2  # token MARK leaves a key that token ASK looks for


def beacon(layer, gain, width=96, vocab=60, positions=512):
    """A one-layer model whose token MARK leaves a value that token ASK picks up: both embeddings are axes of their own, ASK's
    query points along MARK's key.  No position vectors, so the pair means the same everywhere."""
    cfg = config([layer], width=width, vocab=vocab, positions=positions)
    T = lo.random_tensors(cfg, 21)
    T["pos"][:] = 0.0
    T["l0.norm1"][:] = 0.0
    T["embed"][:, :2] = 0.0
    T["embed"][[MARK, ASK]] = 0.0
    axis = {MARK: 0, ASK: 1}
    for t, i in axis.items():
        T["embed"][t, i] = np.sqrt(width)  # after the norm: sqrt(width) along axis i
    m = layer["mixer"]
    H, d = m["heads"], m["dim"]
    e = np.sqrt(width)
    if layer["type"] == "latent_attention":
        c = lo.rms_norm_plain(T["l0.mix.dkv"][:m["kv_rank"], 0] * e, T["l0.mix.dkv.norm"], 1e-5)
        key = (T["l0.mix.uk"] @ c).reshape(H, d)
        T["l0.mix.q"][:, 1] = 0.0
        q = T["l0.mix.q"].reshape(H, d + m["rot_dim"], width)
        q[:, :d, 1] = gain * key / (e * m["scale"] * (key * key).sum(1, keepdims=True))  # score of the pair = gain
    else:
        act = lo.silu if layer["type"] == "lightning" else (lambda z: z)
        T["l0.mix.k"][:, 0] = np.abs(T["l0.mix.k"][:, 0]) * 12.0  # a strong key; positive, so that SiLU keeps it
        T["l0.mix.q"][:, 1] = gain * act(T["l0.mix.k"][:, 0] * e) / e
    return cfg, {n: lo.bf16_round(a) for n, a in T.items()}


def placed(n, marks, asks, vocab=60, seed=5):
    t = np.random.default_rng(seed).integers(3, vocab, n)
    t[list(marks)] = MARK
    t[list(asks)] = ASK
    return t


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [2, 7, 16, 64, 65, 100])
def test_window_edges(cuda, dtype, window):
    cfg, T = beacon(latent(heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=40, window=window), 9.0)
    m = Model(cfg, dtype, tensors=T)
    # one query that just sees its mark, and later one that just misses its own
    p = window + 20
    n = p + window + 5
    tokens = placed(n, [p - window + 1, n - 1 - window], [p, n - 1])
    want = m.oracle(tokens)
    for w in (window - 1, window + 1):  # an edge that is one token off shows in the logits
        off = copy.deepcopy(cfg)
        off["layers"][0]["mixer"]["mask"]["size"] = w
        assert rel(lo.forward(off, m.tensors, tokens), want).max() > 5 * TOL["bfloat16"], w
    check(m.run(tokens), want, dtype)                                        # in a prompt
    check(m.run(tokens, [p] + [1] * (n - p)), want, dtype)                   # decoded
    check(m.run(tokens, [p - 1] + parts(n - p + 1, [2, 3])), want, dtype)    # in short portions
    check(m.run(tokens, [p - window + 2, n - p - 5, window - 3 + 6] if window > 2 else [p, 2, n - p - 2]), want, dtype)  # the mark ends a portion
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["retention", "lightning"])
def test_far_keys_and_chunk_edges(cuda, dtype, kind):
    decay = [0.9999, 0.98]
    layer = retention(2, 16, 24, decay=decay, rot=2, base=1e9) if kind == "retention" else lightning(2, 24, 16, decay=decay)
    cfg, T = beacon(layer, 2.0)
    m = Model(cfg, dtype, tensors=T)
    for distance in (1, 63, 64, 65, 127, 128, 129, 300):
        n = distance + 6
        tokens = placed(n, [4], [4 + distance])
        want = m.oracle(tokens)
        without = tokens.copy()
        without[4] = 9
        assert rel(m.oracle(without), want)[4 + distance] > 5 * TOL["bfloat16"], distance  # the mark is seen from there
        check(m.run(tokens), want, dtype)
        check(m.run(tokens, [distance + 3, 1, 1, 1]), want, dtype)
        check(m.run(tokens, [5, distance + 1]), want, dtype)      # the mark ends a portion
        check(m.run(tokens, [4] + parts(distance + 2, [64, 2])), want, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_decay_of_every_head_counts(cuda, dtype):
    layer = lightning(3, 16, 16, decay=[0.5, 0.9, 0.99])
    cfg = config([layer])
    m = Model(cfg, dtype, seed=6)
    tokens = m.tokens(100)
    want = m.oracle(tokens)
    check(m.run(tokens), want, dtype)
    check(m.run(tokens, [60] + [1] * 40), want, dtype)
    swapped = copy.deepcopy(cfg)
    swapped["layers"][0]["mixer"]["decay"] = [0.9, 0.5, 0.99]
    assert rel(lo.forward(swapped, m.tensors, tokens), want).max() > 3 * TOL["bfloat16"]
    m.close()


def test_plain_forms_agree_with_the_fast_ones(cuda, monkeypatch):
    monkeypatch.setenv("KMLL_LAYERED", "plain")
    plain = Model(config(MIXED), "bfloat16", seed=12)
    monkeypatch.delenv("KMLL_LAYERED")
    fast = Model(config(MIXED), "bfloat16", tensors=plain.tensors)
    tokens = plain.tokens(130)
    want = plain.oracle(tokens)
    for cut in ([130], [100] + [1] * 30):
        check(plain.run(tokens, cut), want, "bfloat16")
        check(fast.run(tokens, cut), want, "bfloat16")
    plain.close()
    fast.close()


# ---- generation through the session layer -----------------------------------------------------------------------------------
@pytest.fixture
def model_dir(tmp_path):
    cfg = config(MIXED)
    T = lo.random_tensors(cfg, 14)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), {n: (np.ascontiguousarray(a).view(np.uint32) >> 16).astype(np.uint16) for n, a in T.items()})
    return str(tmp_path), cfg, T


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation(cuda, model_dir, dtype):
    path, cfg, T = model_dir
    s = Session(registry.load_model(path, dtype, max_seq_len=160))
    prompt = np.random.default_rng(6).integers(0, cfg["vocab"], 45)
    res = s.run_generation_request(prompt, GenerationOptions(max_new_tokens=40))
    gen = res["generated_tokens"]
    assert len(gen) == 40 and res["finish_reason"] == ("max-new-tokens", None) and res["backend"].startswith("bf16")
    mem = res["memory_stats"]
    assert mem["weights_bytes"] > 0 and mem["kv_cache_bytes"] > 0
    # the oracle, fed the same tokens, prefers each of them (within its tolerance where two are close)
    want = lo.forward(cfg, T, np.concatenate([prompt, gen]))
    scale = np.sqrt((want * want).mean())
    for i, t in enumerate(gen):
        row = want[len(prompt) + i - 1]
        assert row.max() - row[t] <= 6 * TOL[dtype] * scale, i
    # a stop token ends the run whatever the size of the device-resident chunks, and the sequence goes on from there
    stop = gen[17]
    first = gen.index(stop)
    for chunk in (16, 7, 1):
        s.CHUNK = chunk
        s.prefill(prompt)
        steps = s.generate_greedy_until(40, 1, stop)
        assert [x.token_id for x in steps] == gen[:first + 1]
        more = s.generate_greedy_until(5)
        assert [x.token_id for x in more] == gen[first + 1:first + 6]
    # the k-best loop and cold sampling take the same tokens; the logits are those of the decode steps
    s.prefill(prompt)
    assert [x.token_id for x in s.generate_greedy_until(8, 3)] == gen[:8]
    s.prefill(prompt)
    assert [x.token_id for x in s.generate_sampled_top_k_until(8, 4, None, SamplingOptions(temperature=0.0))] == gen[:8]
    logits = s.next_logits_to_host()
    assert rel(logits[None].astype(np.float64), want[len(prompt) + 7][None]).max() <= 2 * TOL[dtype]
    # a prompt in portions generates the same
    s.reset_sequence()
    s.extend(prompt[:20])
    s.extend(prompt[20:])
    assert [x.token_id for x in s.generate_greedy_until(10)] == gen[:10]
    with pytest.raises(KmllError):
        s.run_generation_request(prompt, GenerationOptions(max_new_tokens=200))
    s.dec.close()


def test_rewind_replays_the_states(cuda):
    m = Model(config(MIXED), "float32", seed=15, max_seq_len=200)
    tokens = m.tokens(60)
    m.dec.prefill(tokens)
    toks, _ = m.dec.generate_greedy(20)
    seq = np.concatenate([tokens, toks])
    want = m.oracle(seq)
    for position in (75, 60, 33):  # behind the remembered state, at it, ahead of it (the whole prompt is replayed)
        m.dec.rewind(position)
        assert m.dec.position == position
        check(m.dec.extend(seq[position:position + 5], range(5)), want[position:position + 5], "float32")
        m.dec.prefill(tokens)
        m.dec.generate_greedy(20)
    h, _ = m.dec.history(0, 20)
    assert list(h) == list(toks)
    m.close()


def test_limits_are_errors(cuda):
    m = Model(config([lightning()], positions=40), "bfloat16")
    with pytest.raises(KmllError):
        m.dec.extend(m.tokens(41))
    with pytest.raises(KmllError):
        m.dec.extend([m.cfg["vocab"]])
    with pytest.raises(KmllError):
        m.dec.extend([1, 2], [1, 0])
    with pytest.raises(KmllError):
        rt.BatchDecoder(m.dec, 2)
    with pytest.raises(KmllError):
        m.dec.prefill(m.tokens(5), token_loop=True)
    m.dec.reset()
    assert m.dec.extend(m.tokens(40), [39]).shape == (1, m.cfg["vocab"])
    with pytest.raises(KmllError):
        m.dec.extend([1])
    missing = rt.LayeredDecoder(pefisun.layered_config(m.cfg))
    with pytest.raises(KmllError):
        missing.extend([1])  # no weights
    with pytest.raises(KmllError):
        missing.set_tensor(0, rt.T_UK, np.zeros((1, 1), np.uint16))
    assert load().kmll_decoder_init_random(missing._h, 3, 0.05, 1) == 0
    assert np.isfinite(missing.extend(m.tokens(20), [19])).all()
    back = m.dec.get_tensor(0, rt.T_WQ)
    np.testing.assert_array_equal(back, (m.tensors["l0.mix.q"].view(np.uint32) >> 16).astype(np.uint16))
    missing.close()
    m.close()


def test_uniform_decoder_extends_by_decode_steps(cuda):
    cfg = rt.DecoderConfig(dim=256, n_layers=2, n_heads=4, n_kv_heads=2, head_dim=64, hidden_dim=512, vocab_size=640, max_seq_len=64, format=rt.FORMAT_RS_I8)
    dec = rt.Decoder(cfg)
    dec.init_random(3, 0.05)
    t = np.random.default_rng(1).integers(0, 640, 12)
    s = Session(dec)
    got = s.extend(t[:7], [6])
    got2 = s.extend(t[7:], [0, 4])
    ref = Session(dec)
    for n, row in ((7, got[0]), (8, got2[0]), (12, got2[1])):
        ref.prefill(t[:n])
        np.testing.assert_allclose(row, ref.next_logits_to_host(), atol=2e-3)
    dec.close()


# ---- operators through the C ABI --------------------------------------------------------------------------------------------
def test_bf16_linear_operators(cuda):
    import torch

    from kmll_b200 import ops
    gen = torch.Generator(device="cuda").manual_seed(9)

    def randn(*shape):
        return torch.randn(shape, generator=gen, device="cuda")

    ws = ops.linear_batched_bf16_workspace()
    for batch, rows, cols in ((1, 5, 8), (3, 130, 72), (17, 200, 520), (40, 1000, 2056), (64, 128, 4096), (256, 384, 1024), (300, 1300, 320), (700, 96, 64)):
        w = (randn(rows, cols) / cols ** 0.5).bfloat16()
        x, res = randn(batch, cols), randn(batch, rows)
        want = x.bfloat16().double() @ w.double().T + res.double()
        for workspace in (None, ws, ws):
            got = ops.linear_batched_bf16(x.bfloat16(), w, residual=res, workspace=workspace)
            assert float((got.double() - want).abs().max()) <= 2e-5 * cols ** 0.5, (batch, rows, cols)
        got = ops.linear_batched_bf16(x.bfloat16(), w, out_bf16=True, workspace=ws)
        assert float((got.double() - (want - res.double())).abs().max()) <= 0.03
        want = x.double() @ w.double().T + res.double()
        assert float((ops.linear_batched_bf16(x, w, residual=res).double() - want).abs().max()) <= 1e-5 * cols ** 0.5
        norm = randn(cols).bfloat16()
        xd, w0 = x[0].double(), w.double()
        got = ops.linear_bf16(x[0].contiguous(), w, residual=res[0].contiguous())
        assert float((got.double() - (w0 @ xd + res[0].double())).abs().max()) <= 1e-5 * cols ** 0.5
        n = torch.from_numpy(lo.rms_norm_zero_centred(xd.cpu().numpy(), norm.double().cpu().numpy(), 1e-3)).cuda()
        y = w0 @ n
        y[:rows // 2] = y[:rows // 2] * torch.sigmoid(y[:rows // 2])
        got = ops.linear_bf16(x[0].contiguous(), w, norm_weight=norm, norm_offset=1.0, eps=1e-3, silu_rows=rows // 2)
        assert float((got.double() - y).abs().max()) <= 4e-5 * cols ** 0.5
        coef = randn(4).bfloat16()
        n = torch.from_numpy(lo.poly_norm(xd.cpu().numpy(), coef.double().cpu().numpy(), 1e-3)).cuda()
        got = ops.polynorm_linear_bf16(x[0].contiguous(), coef, 1e-3, w)
        assert float((got.double() - w0 @ n).abs().max()) <= 6e-5 * cols ** 0.5
        gate = randn(cols)
        o = xd.cpu().numpy()
        n = lo.rms(o.reshape(-1, 8), 1e-3).reshape(-1) * lo.silu(gate.double().cpu().numpy())
        got = ops.gated_linear_bf16(x[0].contiguous(), gate, w, 1e-3, head_len=8)
        assert float((got.double() - w0 @ torch.from_numpy(n).cuda()).abs().max()) <= 4e-5 * cols ** 0.5
        n = lo.rms_norm_plain(o, norm.double().cpu().numpy(), 1e-3) * lo.sigmoid(gate.double().cpu().numpy())
        got = ops.gated_linear_bf16(x[0].contiguous(), gate, w, 1e-3, norm_weight=norm, sigmoid=True)
        assert float((got.double() - w0 @ torch.from_numpy(n).cuda()).abs().max()) <= 4e-5 * cols ** 0.5
